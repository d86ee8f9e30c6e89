// Layers of a mixed stack (RWKV-style time mixing, retention, latent attention; dense gated feed-forward):
// weights, per-run state and the launches of a step.  The decoder (decoder.inc) owns the step itself -
// token and position hand-over, graphs, LM-head argmax, timing - and calls in here for the layers.
#pragma once
#include <string>
#include <vector>

#include "state.hpp"

namespace rnb {

struct DenseMat {
    uint16_t *w = nullptr;   // bf16 [rows][cols]
    int rows = 0, cols = 0;
    alignas(64) unsigned long long map[16] = {};   // tiled-copy descriptor (64 columns x 64 rows per box)
    bool tiled = false;                            // map is valid: rows are 16-byte aligned
};

struct StackLayer {
    rnb_b200_mixer_cfg c;
    std::vector<float> decay_host;
    float *norm1 = nullptr, *norm1b = nullptr, *norm2 = nullptr, *norm2b = nullptr;
    DenseMat r, k, v, g, w1, w2, w2x /* [w2 | w2] */, q, dkv, uk, uv, o, gate, up, down;
    float *mu = nullptr, *w0 = nullptr, *u = nullptr, *head_norm = nullptr, *dkv_norm = nullptr, *decay = nullptr;
    const void *rot_table = nullptr;   // float2 [max_ctx][dims / 2]
};

// One execution of a layer in a step; a looped layer has one per pass, each with its own state.
struct LayerRun {
    int layer = 0;
    bool add_embedding = false;
    float *state = nullptr, *shift = nullptr, *shift_out = nullptr;   // recurrent state, last normed input
    void *cache = nullptr;                                           // latent rows [max_ctx][ld]
};

struct StackScratch {
    int cap = 0;   // tokens
    float *x[2] = {nullptr, nullptr}, *emb = nullptr, *y = nullptr, *z = nullptr, *w = nullptr, *o = nullptr, *qf = nullptr, *part = nullptr, *starts = nullptr,
          *decays = nullptr, *logits = nullptr;
    uint16_t *th = nullptr;   // tanh of the low-rank decay input as bf16 hi + lo
    void *h = nullptr, *p[4] = {nullptr, nullptr, nullptr, nullptr}, *act = nullptr;
    uint16_t *kn = nullptr, *vx = nullptr;
    int *rows = nullptr;
    uint32_t *tok = nullptr;
    std::vector<void *> allocs;
};

class LayerStack {
public:
    static int create(const rnb_b200_stack_cfg &cfg, const rnb_b200_mixer_cfg *layers, LayerStack **out);
    ~LayerStack();
    int set_tensor(cudaStream_t s, const char *name, uint32_t type, const void *data, const uint64_t *shape, uint32_t n_dims);
    int fill_synthetic(cudaStream_t s, uint64_t seed, float sigma);
    int fill_state_synthetic(cudaStream_t s, int n_pos, uint64_t seed);
    int ready(cudaStream_t s);             // every tensor present, small-step scratch allocated
    int reset(cudaStream_t s);             // a new sequence starts: recurrent states and shifts back to zero
    // All layers for `n` tokens at positions *pos .. *pos + n - 1.  Leaves the residual rows in *x_rows.
    // head (one token): the final norm rides in the last residual pass and logits receive the LM head.
    // trace (host, [runs][n][width]): the residual after every run.
    int forward(cudaStream_t s, const uint32_t *tokens_dev, int n, const int *pos_dev, int pos_host, float **x_rows, float *logits_one, float *trace, int *err);
    // LM head of the residual rows listed in rows_host (n_rows <= piece()), f32 [n_rows][vocab] on the device.
    int head_rows(cudaStream_t s, const float *x, const int *rows_host, int n_rows, float *logits, int *err);
    int piece() const;                      // most tokens of one forward call
    int reserve(int tokens);                // scratch for a forward call of that many tokens
    int time_matvecs(cudaStream_t s, bool count, uint64_t *bytes);   // only the matvec launches of a one-token step
    StackScratch &scratch(int n) { return n <= SMALL ? small_ : big_; }
    uint64_t weight_bytes() const { return weight_bytes_; }
    uint64_t cache_bytes_per_pos() const;
    int n_runs() const { return (int)runs_.size(); }
    float *x_small() const { return small_.x[0]; }
    static constexpr int SMALL = 8;         // up to here tokens go through the matvec kernels

    const rnb_b200_stack_cfg cfg;

private:
    struct Slot {
        std::string name;
        DenseMat *mat = nullptr;
        float **vec = nullptr;
        size_t vec_off = 0, vec_total = 0;   // where in the vector's buffer, and its size
        int64_t rows = 0, cols = 0;          // cols 0: a vector of `rows` values; -1: taken from the tensor
        float synth_mean = 0.f, synth_sigma = 0.f;
        bool set = false;
    };
    struct Mm {
        const DenseMat *w, *w2;
        const void *x;
        size_t ldx;
        void *y;
        bool f32_out;
        const float *decay_bias = nullptr;
    };
    explicit LayerStack(const rnb_b200_stack_cfg &c) : cfg(c) {}
    int init(const rnb_b200_mixer_cfg *layers);
    int alloc(void **p, size_t bytes, std::vector<void *> *owner = nullptr);
    int alloc_scratch(StackScratch &b, int cap);
    int rotation_table(const rnb_b200_rotation &r, const void **out);
    int place(Slot &slot, int64_t rows, int64_t cols);
    void slots_of_layer(int i);
    int matmul(cudaStream_t s, int n, const Mm *jobs, int n_jobs, int *err);
    int boundary(cudaStream_t s, int n, StackScratch &b, int &cur, const float *y, const float *wb, bool emb, const float *wn, const StackLayer *shift, LayerRun *run);
    int mixer_linear(cudaStream_t s, int n, StackScratch &b, StackLayer &L, LayerRun &R, const int *pos_dev, int *err);
    int mixer_latent(cudaStream_t s, int n, StackScratch &b, StackLayer &L, LayerRun &R, const int *pos_dev, int pos_host, int *err);
    bool narrow(int n) const { return n > SMALL && !cfg.f32_math; }   // bf16 activations
    bool absorbed(const StackLayer &L, int n) const;
    int latent_ld(const StackLayer &L) const { return (L.c.kv_rank + L.c.rot_dim + 7) & ~7; }

    std::vector<StackLayer> layers_;
    std::vector<LayerRun> runs_;
    std::vector<Slot> slots_;
    std::vector<void *> allocs_;
    std::vector<std::pair<rnb_b200_rotation, const void *>> tables_;
    DenseMat embed_;
    float *final_norm_ = nullptr;
    StackScratch small_, big_;
    int *counters_ = nullptr;
    bool ready_ = false, loops_ = false;
    uint64_t weight_bytes_ = 0;
    int sm_ = 148, attend_chunks_ = 1;
};

}  // namespace rnb
