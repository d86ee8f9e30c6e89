// Layers of a mixed stack (RWKV-style time mixing, retention, latent attention, gated linear attention, window
// attention, gated delta rule; dense gated feed-forward): weights, per-run state and the launches of a step.  The decoder (decoder.inc) owns the step itself -
// token and position hand-over, graphs, LM-head argmax, timing - and calls in here for the layers.
#pragma once
#include <string>
#include <vector>

#include "state.hpp"

namespace rnb {

struct WindowAttentionArgs;
struct DeltaArgs;

struct DenseMat {
    uint16_t *w = nullptr;   // bf16 [rows][cols]
    int rows = 0, cols = 0;
    alignas(64) unsigned long long map[16] = {};   // tiled-copy descriptor (64 columns x 64 rows per box)
    bool tiled = false;                            // map is valid: rows are 16-byte aligned
};

// A mixer's weights.  Time mixing, retention and latent attention project through one matrix per tensor; the
// others through `in` (their tensors' rows one after the other, at in_at, each padded to 8 rows) and, where
// an f32 result is wanted, `aux`.
struct StackMixer {
    rnb_b200_mixer_cfg c;
    std::string prefix;
    std::vector<float> decay_host;
    DenseMat r, k, v, g, w1, w2, w2x /* [w2 | w2] */, q, dkv, uk, uv, in, aux;
    int in_at[4] = {}, in_rows = 0, aux_rows = 0;
    int act_at = 0, act_cols = 0;      // the output's columns in the input of the layer's output matrix
    float *mu = nullptr, *w0 = nullptr, *u = nullptr, *head_norm = nullptr, *dkv_norm = nullptr, *decay = nullptr, *conv = nullptr, *a_log = nullptr, *dt = nullptr;
    const void *rot_table = nullptr;   // float2 [max_ctx][dims / 2]
};

struct StackLayer {
    std::vector<StackMixer> mixers;
    int n_ff = 0, weights_of = -1;
    int ff_at = 0, out_cols = 0;       // parallel layers: the feed-forward shares the output matrix, from column ff_at on
    float *norm1 = nullptr, *norm1b = nullptr, *norm2 = nullptr, *norm2b = nullptr;
    DenseMat out, gate, up, down;      // out: [width][out_cols], the mixers' output projections (and down) side by side
    bool shifts() const { return mixers[0].c.mixer == RNB_B200_MIXER_WKV; }
};

struct MixerState {
    float *state = nullptr, *shift = nullptr, *shift_out = nullptr;   // recurrent state, last normed input
    void *cache = nullptr;                                           // latent rows [max_ctx][ld]; keys [ring][kv_heads * dim]
    void *values = nullptr;                                          // values [ring][kv_heads * vdim]
    float *conv_ring = nullptr;                                      // last inputs of the short convolutions
};
// One execution of a layer in a step; a looped layer has one per pass, each with its own state.
struct LayerRun {
    int layer = 0;                     // whose weights
    bool add_embedding = false;
    std::vector<MixerState> m;
};

struct StackScratch {
    int cap = 0;   // tokens
    float *x[2] = {nullptr, nullptr}, *emb = nullptr, *y = nullptr, *z = nullptr, *w = nullptr, *o = nullptr, *qf = nullptr, *part = nullptr, *starts = nullptr,
          *decays = nullptr, *logits = nullptr;
    uint16_t *th = nullptr;   // tanh of the low-rank decay input as bf16 hi + lo
    void *h = nullptr, *p[4] = {nullptr, nullptr, nullptr, nullptr}, *act = nullptr, *qn = nullptr;
    float *aux[2] = {nullptr, nullptr};
    uint16_t *kn = nullptr, *vx = nullptr, *cqk = nullptr, *cv = nullptr;
    uint8_t *rec = nullptr;
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
        int64_t row0 = 0, col0 = 0, all_rows = 0, all_cols = 0;   // all_rows > 0: a block of a larger matrix, zeros between the blocks
        float synth_mean = 0.f, synth_sigma = 0.f;
        bool set = false;
    };
    struct Mm {
        const DenseMat *w, *w2;
        const void *x;
        size_t ldx;
        void *y;
        bool f32_out;
        size_t ldy = 0;                      // 0: rows
        const float *decay_bias = nullptr;   // y: decays of the mixer `decay`
        const rnb_b200_mixer_cfg *decay = nullptr;
    };
    explicit LayerStack(const rnb_b200_stack_cfg &c) : cfg(c) {}
    int init(const rnb_b200_mixer_cfg *layers);
    int alloc(void **p, size_t bytes, std::vector<void *> *owner = nullptr);
    int alloc_scratch(StackScratch &b, int cap);
    int rotation_table(const rnb_b200_rotation &r, const void **out);
    int place(cudaStream_t s, Slot &slot, int64_t rows, int64_t cols);
    void slots_of_layer(int i);
    int matmul(cudaStream_t s, int n, const Mm *jobs, int n_jobs, int *err);
    int in_jobs(int n, StackScratch &b, StackLayer &L, Mm *jobs);   // the projections that read the layer's normed input
    Mm out_job(StackScratch &b, StackLayer &L);
    int boundary(cudaStream_t s, int n, StackScratch &b, int &cur, const float *y, const float *wb, bool emb, const float *wn, const float *bn, const StackLayer *shift, LayerRun *run);
    int run_mixer(cudaStream_t s, int n, StackScratch &b, StackLayer &L, int i, MixerState &R, const int *pos_dev, int pos_host, int *err);
    int mixer_linear(cudaStream_t s, int n, StackScratch &b, StackLayer &L, int i, MixerState &R, const int *pos_dev, int *err);
    int mixer_latent(cudaStream_t s, int n, StackScratch &b, StackLayer &L, int i, MixerState &R, const int *pos_dev, int pos_host, int *err);
    int mixer_attention(cudaStream_t s, int n, StackScratch &b, StackLayer &L, int i, MixerState &R, const int *pos_dev);
    WindowAttentionArgs attention_args(int n, StackScratch &b, StackLayer &L, int i, MixerState &R, const int *pos_dev) const;
    DeltaArgs delta_args(int n, StackScratch &b, StackLayer &L, int i, MixerState &R, const int *pos_dev) const;
    int mixers_attention_delta(cudaStream_t s, int n, StackScratch &b, StackLayer &L, LayerRun &R, const int *pos_dev);
    int mixer_delta(cudaStream_t s, int n, StackScratch &b, StackLayer &L, int i, MixerState &R, const int *pos_dev, int *err);
    int head_norm_gate(cudaStream_t s, int n, StackScratch &b, const StackLayer &L, const StackMixer &M, const void *g, int ldg);
    void *act_of(StackScratch &b, const StackMixer &M, int n) const { return (char *)b.act + (size_t)M.act_at * (narrow(n) ? 2 : 4); }
    int attention_ring(const rnb_b200_mixer_cfg &m) const;
    int attention_chunks(const rnb_b200_mixer_cfg &m) const;
    bool attention_tiled(const rnb_b200_mixer_cfg &m) const;
    bool parallel() const { return cfg.block == RNB_B200_BLOCK_PARALLEL; }
    template <class Fn>
    void each_mixer(Fn fn) const {
        for (const StackLayer &L : layers_)
            for (const StackMixer &M : L.mixers) fn(L, M);
    }
    bool narrow(int n) const { return n > SMALL && !cfg.f32_math; }   // bf16 activations
    bool absorbed(const rnb_b200_mixer_cfg &m, int n) const;
    static int latent_ld(const rnb_b200_mixer_cfg &m) { return (m.kv_rank + m.rot_dim + 7) & ~7; }

    std::vector<StackLayer> layers_;
    std::vector<LayerRun> runs_;
    std::vector<Slot> slots_;
    std::vector<void *> allocs_;
    std::vector<std::pair<rnb_b200_rotation, const void *>> tables_;
    DenseMat embed_;
    float *final_norm_ = nullptr, *final_bias_ = nullptr;
    StackScratch small_, big_;
    int *counters_ = nullptr, counters_of_mixer_ = 0;
    bool ready_ = false, loops_ = false;
    uint64_t weight_bytes_ = 0;
    int sm_ = 148, attend_chunks_ = 1;
};

}  // namespace rnb
