// Host side of the mixed stacks: weights by name, per-run state, scratch, and the launch order of a step.
#include "layer_stack.hpp"

#include <cuda.h>
#include <math.h>

#include <algorithm>

#include "delta_rule.cuh"
#include "dense.cuh"
#include "latent_attention.cuh"
#include "launch.hpp"
#include "layer_glue.cuh"
#include "linear_state.cuh"
#include "window_attention.cuh"

namespace rnb {

// ---- synthetic weights (bench) --------------------------------------------------------------------
__device__ __forceinline__ float synth_normal(uint64_t seed, uint64_t i) {
    auto mix = [](uint64_t z) {
        z += 0x9e3779b97f4a7c15ull;
        z = (z ^ (z >> 30)) * 0xbf58476d1ce4e5b9ull;
        z = (z ^ (z >> 27)) * 0x94d049bb133111ebull;
        return z ^ (z >> 31);
    };
    const uint64_t r = mix(seed ^ mix(i));
    const float u1 = ((float)(uint32_t)(r >> 40) + 1.0f) * (1.0f / 16777217.0f), u2 = (float)(uint32_t)(r & 0xffffff) * (1.0f / 16777216.0f);
    return sqrtf(-2.0f * logf(u1)) * cosf(6.2831853f * u2);
}
template <class T>
RNB_GLOBAL void __launch_bounds__(256) synth_dense_kernel(T *out, size_t n, uint64_t seed, float mean, float sigma) {
    pdl_launch_dependents();
    pdl_wait();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) out[i] = from_f32<T>(mean + sigma * synth_normal(seed, i));
}
template <class T>
static int synth_dense(cudaStream_t s, T *out, size_t n, uint64_t seed, float mean, float sigma) {
    if (n) RNB_CU(launch_k(synth_dense_kernel<T>, dim3((unsigned)std::min<size_t>((n + 255) / 256, 8192)), dim3(256), 0, s, out, n, seed, mean, sigma));
    return RNB_B200_OK;
}

// ---- creation -------------------------------------------------------------------------------------
LayerStack::~LayerStack() {
    for (void *p : allocs_) cudaFree(p);
    for (void *p : small_.allocs) cudaFree(p);
    for (void *p : big_.allocs) cudaFree(p);
}

int LayerStack::alloc(void **p, size_t bytes, std::vector<void *> *owner) {
    *p = nullptr;
    const cudaError_t e = cudaMalloc(p, ((bytes + 255) & ~(size_t)255) + 256);
    if (e != cudaSuccess) return fail_cuda(e, "cudaMalloc(stack)");
    (owner ? *owner : allocs_).push_back(*p);
    return RNB_B200_OK;
}

static int round_pow2(int n) {
    int p = 1;
    while (p < n) p *= 2;
    return p;
}

int LayerStack::create(const rnb_b200_stack_cfg &c, const rnb_b200_mixer_cfg *layers, LayerStack **out) {
    LayerStack *st = new LayerStack(c);
    const int rc = st->init(layers);
    if (rc != RNB_B200_OK) {
        delete st;
        return rc;
    }
    *out = st;
    return RNB_B200_OK;
}

static int round8(int n) { return (n + 7) & ~7; }
// time mixing, retention and latent attention keep a matrix per tensor; the others project through StackMixer::in
static bool joined_rows(const rnb_b200_mixer_cfg &m) { return m.mixer == RNB_B200_MIXER_GLA || m.mixer == RNB_B200_MIXER_ATTENTION || m.mixer == RNB_B200_MIXER_DELTA; }
static bool rotates(const rnb_b200_mixer_cfg &m) { return m.mixer == RNB_B200_MIXER_RETENTION || m.mixer == RNB_B200_MIXER_LATENT_ATTENTION || m.mixer == RNB_B200_MIXER_ATTENTION; }
static size_t attention_step_bytes(const rnb_b200_mixer_cfg &m, bool f32) {
    const int rep = m.heads / m.kv_heads;
    return f32 ? attention_step_smem<float>(rep, m.dim, m.vdim).bytes : attention_step_smem<bf16>(rep, m.dim, m.vdim).bytes;
}

static int check_mixer(const rnb_b200_mixer_cfg &m, int i, bool f32) {
    if (m.heads < 1 || m.dim < 1 || m.n_ff < 0) return fail(RNB_B200_VALIDATION_FAILED, "layer %d: invalid mixer shape", i);
    if (m.vdim < 1) return fail(RNB_B200_VALIDATION_FAILED, "layer %d: invalid value size", i);
    const rnb_b200_rotation &r = m.rot;
    const int rotated = m.mixer == RNB_B200_MIXER_LATENT_ATTENTION ? m.rot_dim : m.dim;
    if (rotates(m) && (r.dims < 0 || r.dims % 2 || r.dims > rotated || (r.dims > 0 && !(r.base > 1.0))))
        return fail(RNB_B200_VALIDATION_FAILED, "layer %d: rotation of %d dimensions does not fit %d", i, r.dims, rotated);
    switch (m.mixer) {
    case RNB_B200_MIXER_WKV:
    case RNB_B200_MIXER_RETENTION:
    case RNB_B200_MIXER_GLA:
        if (m.dim > 512) return fail(RNB_B200_UNSUPPORTED, "layer %d: state channels %d exceed 512", i, m.dim);
        if (m.mixer == RNB_B200_MIXER_RETENTION && !m.decay) return fail(RNB_B200_VALIDATION_FAILED, "layer %d: retention needs a decay per head", i);
        if (m.mixer == RNB_B200_MIXER_GLA && !(m.tau > 0.f)) return fail(RNB_B200_VALIDATION_FAILED, "layer %d: tau must be positive", i);
        return RNB_B200_OK;
    case RNB_B200_MIXER_LATENT_ATTENTION:
        if (m.kv_rank < 1 || m.rot_dim < 0) return fail(RNB_B200_VALIDATION_FAILED, "layer %d: invalid latent shape", i);
        if (m.kv_rank + m.rot_dim > 1152) return fail(RNB_B200_UNSUPPORTED, "layer %d: cache row of %d exceeds 1152", i, m.kv_rank + m.rot_dim);
        return RNB_B200_OK;
    case RNB_B200_MIXER_ATTENTION:
    case RNB_B200_MIXER_DELTA:
        if (m.kv_heads < 1 || m.heads % m.kv_heads) return fail(RNB_B200_VALIDATION_FAILED, "layer %d: %d heads do not share %d key heads evenly", i, m.heads, m.kv_heads);
        if (m.mixer == RNB_B200_MIXER_ATTENTION) {
            if (m.window < 0) return fail(RNB_B200_VALIDATION_FAILED, "layer %d: window of %d", i, m.window);
            if (attention_step_bytes(m, f32) > 220 * 1024) return fail(RNB_B200_UNSUPPORTED, "layer %d: %d heads on %d key heads of %d / %d do not fit an SM", i, m.heads, m.kv_heads, m.dim, m.vdim);
        } else {
            if (m.conv < 1) return fail(RNB_B200_VALIDATION_FAILED, "layer %d: convolutions of %d taps", i, m.conv);
            if (m.dim > 512) return fail(RNB_B200_UNSUPPORTED, "layer %d: state channels %d exceed 512", i, m.dim);
        }
        return RNB_B200_OK;
    default:
        return fail(RNB_B200_UNSUPPORTED, "layer %d: unknown mixer %d", i, m.mixer);
    }
}

static bool same_shape(const StackLayer &a, const StackLayer &b) {
    if (a.n_ff != b.n_ff || a.mixers.size() != b.mixers.size()) return false;
    for (size_t i = 0; i < a.mixers.size(); i++) {
        const rnb_b200_mixer_cfg &x = a.mixers[i].c, &y = b.mixers[i].c;
        if (x.mixer != y.mixer || x.heads != y.heads || x.kv_heads != y.kv_heads || x.dim != y.dim || x.vdim != y.vdim || x.rot_dim != y.rot_dim ||
            x.kv_rank != y.kv_rank || x.window != y.window || x.conv != y.conv)
            return false;
    }
    return true;
}

int LayerStack::init(const rnb_b200_mixer_cfg *layers) {
    const rnb_b200_stack_cfg &c = cfg;
    if (c.n_layer < 1 || c.width < 1 || c.vocab < 1 || c.max_ctx < 1) return fail(RNB_B200_VALIDATION_FAILED, "stack: invalid shape");
    if (c.width > 24576) return fail(RNB_B200_UNSUPPORTED, "stack: width %d exceeds 24576", c.width);
    if (c.norm == RNB_B200_NORM_LAYER && !parallel()) return fail(RNB_B200_UNSUPPORTED, "stack: sandwich layers have root-mean-square norms");
    sm_ = state().sm_count;
    for (int k = 0; k < c.n_layer; k++) {
        const bool join = layers[k].join != 0;
        if (join && (layers_.empty() || layers_.back().mixers.size() != 1 || !joined_rows(layers[k]) || !joined_rows(layers_.back().mixers[0].c)))
            return fail(RNB_B200_UNSUPPORTED, "stack: record %d cannot join the layer before it", k);
        if (!join) layers_.emplace_back();
        StackLayer &L = layers_.back();
        const int i = (int)layers_.size() - 1;
        if (!join) L.n_ff = layers[k].n_ff, L.weights_of = layers[k].weights_of;
        L.mixers.emplace_back();
        StackMixer &M = L.mixers.back();
        M.c = layers[k];
        M.prefix = layers[k].prefix ? layers[k].prefix : "mix.";
        if (M.c.mixer == RNB_B200_MIXER_WKV) M.c.vdim = M.c.dim;
        RNB_TRY(check_mixer(M.c, i, c.f32_math != 0));
        if (M.c.mixer == RNB_B200_MIXER_WKV && parallel()) return fail(RNB_B200_UNSUPPORTED, "layer %d: time mixing has inputs of its own and cannot share a norm", i);
        if (M.c.mixer == RNB_B200_MIXER_RETENTION)
            for (int h = 0; h < M.c.heads; h++) M.decay_host.push_back((float)M.c.decay[h]);
        M.c.decay = nullptr;
        M.c.prefix = nullptr;
    }
    const int n_layer = (int)layers_.size();
    loops_ = c.loop_times > 1;
    if (loops_ && (c.loop_start < 0 || c.loop_stop <= c.loop_start || c.loop_stop > n_layer)) return fail(RNB_B200_VALIDATION_FAILED, "stack: invalid loop %d .. %d", c.loop_start, c.loop_stop);
    std::vector<int> weights((size_t)n_layer);   // whose tensors a layer uses
    for (int i = 0; i < n_layer; i++) {
        int j = i;
        for (int hops = 0; j >= 0 && j < n_layer && layers_[j].weights_of >= 0 && hops <= n_layer; hops++) j = layers_[j].weights_of;
        if (j < 0 || j >= n_layer || layers_[j].weights_of >= 0 || !same_shape(layers_[i], layers_[j]))
            return fail(RNB_B200_VALIDATION_FAILED, "layer %d cannot use the weights of layer %d", i, layers_[i].weights_of);
        weights[i] = j;
    }
    for (int i = 0; i < n_layer; i++) {
        StackLayer &L = layers_[i];
        if (weights[i] != i) continue;
        for (StackMixer &M : L.mixers) {
            if (!M.decay_host.empty()) {
                RNB_TRY(alloc((void **)&M.decay, M.decay_host.size() * 4));
                RNB_CU(cudaMemcpy(M.decay, M.decay_host.data(), M.decay_host.size() * 4, cudaMemcpyHostToDevice));
            }
            if (rotates(M.c) && M.c.rot.dims > 0) RNB_TRY(rotation_table(M.c.rot, &M.rot_table));
        }
        slots_of_layer(i);
    }
    Slot e;
    e.name = "embed", e.mat = &embed_, e.rows = c.vocab, e.cols = c.width;
    slots_.push_back(e);
    Slot f;
    f.name = "final.norm", f.vec = &final_norm_, f.rows = f.vec_total = c.width, f.synth_mean = c.norm == RNB_B200_NORM_LAYER ? 1.f : 0.f;
    slots_.push_back(f);
    if (c.norm == RNB_B200_NORM_LAYER) {
        f.name = "final.norm.b", f.vec = &final_bias_, f.synth_mean = 0.f;
        slots_.push_back(f);
    }
    const int a = loops_ ? c.loop_start : 0, b = loops_ ? c.loop_stop : 0, times = loops_ ? c.loop_times : 0;
    auto push = [&](int layer, bool emb) {
        LayerRun r;
        r.layer = weights[layer];
        r.add_embedding = emb;
        runs_.push_back(r);
    };
    for (int i = 0; i < a; i++) push(i, false);
    for (int t = 0; t < times; t++)
        for (int i = a; i < b; i++) push(i, t > 0 && i == a);
    for (int i = b; i < n_layer; i++) push(i, false);
    int counters = 1;
    const size_t cs = c.f32_math ? 4 : 2;
    for (LayerRun &r : runs_)
        for (const StackMixer &M : layers_[r.layer].mixers) {
            const rnb_b200_mixer_cfg &m = M.c;
            counters = std::max(counters, m.mixer == RNB_B200_MIXER_ATTENTION ? SMALL * m.kv_heads : m.heads);
            MixerState st;
            if (m.mixer == RNB_B200_MIXER_LATENT_ATTENTION) {
                RNB_TRY(alloc(&st.cache, (size_t)c.max_ctx * latent_ld(m) * cs));
            } else if (m.mixer == RNB_B200_MIXER_ATTENTION) {
                RNB_TRY(alloc(&st.cache, (size_t)attention_ring(m) * m.kv_heads * m.dim * cs));
                RNB_TRY(alloc(&st.values, (size_t)attention_ring(m) * m.kv_heads * m.vdim * cs));
            } else {
                RNB_TRY(alloc((void **)&st.state, (size_t)m.heads * m.dim * m.vdim * 4));
                if (m.mixer == RNB_B200_MIXER_WKV) {
                    RNB_TRY(alloc((void **)&st.shift, (size_t)c.width * 4));
                    RNB_TRY(alloc((void **)&st.shift_out, (size_t)c.width * 4));
                }
                if (m.mixer == RNB_B200_MIXER_DELTA) RNB_TRY(alloc((void **)&st.conv_ring, (size_t)delta_ring_rows(m.conv) * (2 * m.kv_heads * m.dim + m.heads * m.vdim) * 4));
            }
            r.m.push_back(st);
        }
    counters_of_mixer_ = counters;   // two mixers may run in one launch
    RNB_TRY(alloc((void **)&counters_, (size_t)2 * counters * 4));
    RNB_CU(cudaMemset(counters_, 0, (size_t)2 * counters * 4));
    RNB_CU(cudaStreamSynchronize(nullptr));
    attend_chunks_ = std::max(1, std::min((c.max_ctx + 127) / 128, 64));
    return RNB_B200_OK;
}

// Rows of an attention mixer's key and value rings: what a query sees beside the tokens of one forward call.
int LayerStack::attention_ring(const rnb_b200_mixer_cfg &m) const { return m.window > 0 ? (int)std::min<int64_t>(cfg.max_ctx, (int64_t)m.window - 1 + piece()) : cfg.max_ctx; }
// CTAs that share the keys of a step: 64 keys or more each, about two CTAs per SM
int LayerStack::attention_chunks(const rnb_b200_mixer_cfg &m) const {
    const int seen = m.window > 0 ? std::min(m.window, cfg.max_ctx) : cfg.max_ctx;
    return std::max(1, std::min({(seen + AS_KEYS - 1) / AS_KEYS, AS_KEYS, std::max(1, 2 * sm_ / m.kv_heads)}));
}
bool LayerStack::attention_tiled(const rnb_b200_mixer_cfg &m) const {
    return !cfg.f32_math && causal_attention_vcols(m.vdim) && causal_attention_smem(m.dim, m.vdim) <= 227 * 1024;
}

// cos and sin of position * frequency for every position, computed in binary64 and rounded once.
int LayerStack::rotation_table(const rnb_b200_rotation &r, const void **out) {
    for (auto &t : tables_)
        if (!memcmp(&t.first, &r, sizeof(r))) {
            *out = t.second;
            return RNB_B200_OK;
        }
    const int half = r.dims / 2;
    std::vector<double> f((size_t)half);
    double mult = 1.0, lo = 0.0, hi = 0.0;
    if (r.scaled == RNB_B200_ROTATION_YARN) {
        auto dim_of = [&](double turns) { return r.dims * log(r.original / (2.0 * M_PI * turns)) / (2.0 * log(r.base)); };
        lo = std::max(floor(dim_of(r.fast)), 0.0);
        hi = std::min(ceil(dim_of(r.slow)), (double)r.dims - 1.0);
        mult = 0.1 * log(r.factor) + 1.0;
    }
    for (int i = 0; i < half; i++) {
        f[i] = pow(r.base, -2.0 * i / r.dims);
        if (r.scaled == RNB_B200_ROTATION_LINEAR) f[i] /= r.factor;
        if (r.scaled == RNB_B200_ROTATION_YARN) {
            const double ramp = std::min(std::max((i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
            f[i] = f[i] / r.factor * ramp + f[i] * (1.0 - ramp);
        }
    }
    std::vector<float> tab((size_t)cfg.max_ctx * r.dims);
    for (int p = 0; p < cfg.max_ctx; p++)
        for (int i = 0; i < half; i++) {
            tab[((size_t)p * half + i) * 2] = (float)(cos(p * f[i]) * mult);
            tab[((size_t)p * half + i) * 2 + 1] = (float)(sin(p * f[i]) * mult);
        }
    void *dev = nullptr;
    RNB_TRY(alloc(&dev, tab.size() * 4));
    RNB_CU(cudaMemcpy(dev, tab.data(), tab.size() * 4, cudaMemcpyHostToDevice));
    tables_.push_back({r, dev});
    *out = dev;
    return RNB_B200_OK;
}

// ---- weights --------------------------------------------------------------------------------------
void LayerStack::slots_of_layer(int i) {
    StackLayer &L = layers_[i];
    const int64_t D = cfg.width;
    const std::string p = "l" + std::to_string(i) + ".";
    auto mat = [&](const std::string &name, DenseMat *dst, int64_t rows, int64_t cols) -> Slot & {
        Slot s;
        s.name = name, s.mat = dst, s.rows = rows, s.cols = cols;
        slots_.push_back(s);
        return slots_.back();
    };
    auto vec = [&](const std::string &name, float **dst, int64_t n, float mean = 0.f, float sigma = 0.f, size_t off = 0, size_t total = 0) {
        Slot s;
        s.name = name, s.vec = dst, s.rows = n, s.vec_off = off, s.vec_total = total ? total : (size_t)n, s.synth_mean = mean, s.synth_sigma = sigma;
        slots_.push_back(s);
    };
    const bool ln = cfg.norm == RNB_B200_NORM_LAYER;
    vec(p + "norm1", &L.norm1, D, ln ? 1.f : 0.f);
    if (ln) vec(p + "norm1.b", &L.norm1b, D);
    if (!parallel()) vec(p + "norm1b", &L.norm1b, D);
    int at = 0;
    for (StackMixer &M : L.mixers) {
        M.act_at = at;
        M.act_cols = M.c.heads * M.c.vdim;
        at = round8(at + M.act_cols);
    }
    L.ff_at = at;
    L.out_cols = parallel() && L.n_ff > 0 ? round8(at + L.n_ff) : at;
    for (StackMixer &M : L.mixers) {
        const rnb_b200_mixer_cfg &m = M.c;
        const int64_t hd = (int64_t)m.heads * m.dim, hv = (int64_t)m.heads * m.vdim, rank = m.decay_rank > 0 ? m.decay_rank : -1;
        const std::string x = p + M.prefix;
        Slot &o = mat(x + "o", &L.out, D, hv);
        o.all_rows = D, o.all_cols = L.out_cols, o.col0 = M.act_at;
        // tensors that share the matrix `in`: (name, rows)
        auto rows_of_in = [&](std::initializer_list<std::pair<const char *, int64_t>> parts) {
            int n = 0;
            M.in_rows = 0;
            for (auto &q : parts) M.in_at[n++] = M.in_rows, M.in_rows += round8((int)q.second);
            n = 0;
            for (auto &q : parts) {
                Slot &s = mat(x + q.first, &M.in, q.second, D);
                s.all_rows = M.in_rows, s.all_cols = D, s.row0 = M.in_at[n++];
            }
        };
        auto rows_of_aux = [&](std::initializer_list<const char *> names) {
            M.aux_rows = (int)names.size() * m.heads;
            int n = 0;
            for (const char *q : names) {
                Slot &s = mat(x + q, &M.aux, m.heads, D);
                s.all_rows = M.aux_rows, s.all_cols = D, s.row0 = (int64_t)m.heads * n++;
            }
        };
        if (m.mixer == RNB_B200_MIXER_WKV) {
            const char *mix = "rkvgw";
            for (int j = 0; j < 5; j++) vec(x + "mu." + mix[j], &M.mu, D, 0.5f, 0.1f, (size_t)j * D, (size_t)5 * D);
            mat(x + "r", &M.r, hd, D);
            mat(x + "k", &M.k, hd, D);
            mat(x + "v", &M.v, hd, D);
            mat(x + "g", &M.g, hd, D);
            mat(x + "w1", &M.w1, rank, D);
            mat(x + "w2", &M.w2, hd, rank);
            vec(x + "w0", &M.w0, hd, -1.5f, 1.0f);
            vec(x + "u", &M.u, hd, 0.f, 0.5f);
            vec(x + "norm", &M.head_norm, hd, 1.f);
        } else if (m.mixer == RNB_B200_MIXER_RETENTION) {
            mat(x + "q", &M.q, hd, D);
            mat(x + "k", &M.k, hd, D);
            mat(x + "v", &M.v, hv, D);
            mat(x + "g", &M.g, hv, D);
        } else if (m.mixer == RNB_B200_MIXER_LATENT_ATTENTION) {
            mat(x + "q", &M.q, (int64_t)m.heads * (m.dim + m.rot_dim), D);
            mat(x + "dkv", &M.dkv, m.kv_rank + m.rot_dim, D);
            vec(x + "dkv.norm", &M.dkv_norm, m.kv_rank, 1.f);
            mat(x + "uk", &M.uk, hd, m.kv_rank);
            mat(x + "uv", &M.uv, hv, m.kv_rank);
        } else if (m.mixer == RNB_B200_MIXER_GLA) {
            rows_of_in({{"q", hd}, {"k", hd}, {"v", hv}, {"g", hv}});
            mat(x + "a1", &M.w1, rank, D);
            mat(x + "a2", &M.w2, hd, rank);
            vec(x + "a2.b", &M.w0, hd, 2.f, 1.f);
            vec(x + "norm", &M.head_norm, m.vdim, 1.f);
        } else if (m.mixer == RNB_B200_MIXER_ATTENTION) {
            rows_of_in({{"q", hd}, {"k", (int64_t)m.kv_heads * m.dim}, {"v", (int64_t)m.kv_heads * m.vdim}});
            if (m.head_gate) rows_of_aux({"g"});
        } else {
            const int64_t qc = (int64_t)m.kv_heads * m.dim;
            const size_t taps = (size_t)m.conv, all = (size_t)(2 * qc + hv) * taps;
            rows_of_in({{"q", qc}, {"k", qc}, {"v", hv}, {"g", hv}});
            rows_of_aux({"b", "a"});
            vec(x + "q.conv", &M.conv, qc * m.conv, 0.f, 0.5f, 0, all);
            vec(x + "k.conv", &M.conv, qc * m.conv, 0.f, 0.5f, (size_t)qc * taps, all);
            vec(x + "v.conv", &M.conv, hv * m.conv, 0.f, 0.5f, (size_t)2 * qc * taps, all);
            vec(x + "A_log", &M.a_log, m.heads, 0.f, 0.5f);
            vec(x + "dt_bias", &M.dt, m.heads, -2.f, 1.f);
            vec(x + "norm", &M.head_norm, m.vdim, 1.f);
        }
    }
    if (L.n_ff > 0) {
        if (!parallel()) {
            vec(p + "norm2", &L.norm2, D);
            vec(p + "norm2b", &L.norm2b, D);
        }
        mat(p + "mlp.gate", &L.gate, L.n_ff, D);
        mat(p + "mlp.up", &L.up, L.n_ff, D);
        Slot &d = mat(p + "mlp.down", parallel() ? &L.out : &L.down, D, L.n_ff);
        if (parallel()) d.all_rows = D, d.all_cols = L.out_cols, d.col0 = L.ff_at;
    }
}

// Device storage of a tensor; rows / cols as the tensor has them.  A slot that is a block of a larger matrix
// places the whole matrix.
int LayerStack::place(cudaStream_t s, Slot &slot, int64_t rows, int64_t cols) {
    if (slot.vec) {
        if (!*slot.vec) {
            RNB_TRY(alloc((void **)slot.vec, slot.vec_total * 4));
            weight_bytes_ += slot.vec_total * 4;
        }
        return RNB_B200_OK;
    }
    DenseMat &m = *slot.mat;
    if (!m.w) weight_bytes_ += slot.all_rows ? 0 : (uint64_t)rows * cols * 2;
    if (slot.all_rows) weight_bytes_ += slot.set ? 0 : (uint64_t)rows * cols * 2, rows = slot.all_rows, cols = slot.all_cols;
    if (!m.w) {
        RNB_TRY(alloc((void **)&m.w, (size_t)rows * cols * 2));
        if (slot.all_rows) RNB_CU(cudaMemsetAsync(m.w, 0, (size_t)rows * cols * 2, s));
    }
    m.rows = (int)rows;
    m.cols = (int)cols;
    m.tiled = cols % 8 == 0;
    if (m.tiled) {
        PgTensorMap t;
        RNB_TRY(encode_token_map(&t, m.w, (size_t)rows, (size_t)cols, (size_t)cols, 64));
        memcpy(m.map, &t, sizeof(m.map));
    }
    return RNB_B200_OK;
}

int LayerStack::set_tensor(cudaStream_t s, const char *name, uint32_t type, const void *data, const uint64_t *shape, uint32_t n_dims) {
    Slot *slot = nullptr;
    for (Slot &t : slots_)
        if (t.name == name) slot = &t;
    if (!slot) return fail(RNB_B200_UNSUPPORTED, "stack has no tensor '%s'", name);
    if (ready_) return fail(RNB_B200_VALIDATION_FAILED, "stack: weights cannot change once it runs");
    uint64_t n = 1;
    for (uint32_t i = 0; i < n_dims; i++) n *= shape[i];
    if (slot->vec) {
        if (n != (uint64_t)slot->rows) return fail(RNB_B200_VALIDATION_FAILED, "tensor '%s': %llu values, expected %lld", name, (unsigned long long)n, (long long)slot->rows);
        if (type != 0 && type != 30) return fail(RNB_B200_UNSUPPORTED, "tensor '%s': type %u (BF16 or F32 expected)", name, type);
        RNB_TRY(place(s, *slot, slot->rows, 0));
        std::vector<float> f((size_t)n);
        if (type == 0) memcpy(f.data(), data, n * 4);
        else
            for (uint64_t i = 0; i < n; i++) {
                uint16_t h;
                memcpy(&h, (const uint8_t *)data + 2 * i, 2);
                const uint32_t b = (uint32_t)h << 16;
                memcpy(&f[i], &b, 4);
            }
        RNB_CU(cudaMemcpy(*slot->vec + slot->vec_off, f.data(), n * 4, cudaMemcpyHostToDevice));
    } else {
        if (n_dims != 2 || (slot->rows >= 0 && shape[0] != (uint64_t)slot->rows) || (slot->cols >= 0 && shape[1] != (uint64_t)slot->cols) || n == 0)
            return fail(RNB_B200_VALIDATION_FAILED, "tensor '%s': shape does not match the configuration (%lld x %lld expected)", name, (long long)slot->rows, (long long)slot->cols);
        if (type != 30) return fail(RNB_B200_UNSUPPORTED, "tensor '%s': matrices must be BF16 (type %u found)", name, type);
        RNB_TRY(place(s, *slot, (int64_t)shape[0], (int64_t)shape[1]));
        const DenseMat &m = *slot->mat;
        RNB_CU(cudaMemcpy2DAsync(m.w + (size_t)slot->row0 * m.cols + slot->col0, (size_t)m.cols * 2, data, (size_t)shape[1] * 2, (size_t)shape[1] * 2, (size_t)shape[0],
                                 cudaMemcpyHostToDevice, s));
        RNB_CU(cudaStreamSynchronize(s));
    }
    slot->set = true;
    return RNB_B200_OK;
}

int LayerStack::fill_synthetic(cudaStream_t s, uint64_t seed, float sigma) {
    uint64_t id = seed * 1000003ull;
    for (Slot &t : slots_) {
        const int64_t rows = t.rows < 0 ? 64 : t.rows, cols = t.cols < 0 ? 64 : t.cols;
        RNB_TRY(place(s, t, rows, cols));
        if (t.vec) RNB_TRY(synth_dense<float>(s, *t.vec + t.vec_off, (size_t)rows, ++id, t.synth_mean, t.synth_sigma));
        else if (!t.all_rows || cols == t.all_cols) RNB_TRY(synth_dense<bf16>(s, reinterpret_cast<bf16 *>(t.mat->w) + (size_t)t.row0 * t.mat->cols, (size_t)rows * cols, ++id, 0.f, sigma));
        else {   // columns of a wider matrix
            std::vector<void *> tmp;
            void *d = nullptr;
            RNB_TRY(alloc(&d, (size_t)rows * cols * 2, &tmp));
            const int rc = synth_dense<bf16>(s, reinterpret_cast<bf16 *>(d), (size_t)rows * cols, ++id, 0.f, sigma);
            const cudaError_t e = cudaMemcpy2DAsync(t.mat->w + (size_t)t.row0 * t.mat->cols + t.col0, (size_t)t.mat->cols * 2, d, (size_t)cols * 2, (size_t)cols * 2, (size_t)rows,
                                                    cudaMemcpyDeviceToDevice, s);
            cudaStreamSynchronize(s);
            cudaFree(d);
            RNB_TRY(rc);
            if (e != cudaSuccess) return fail_cuda(e, "cudaMemcpy2DAsync");
        }
        t.set = true;
    }
    RNB_CU(cudaStreamSynchronize(s));
    return RNB_B200_OK;
}

int LayerStack::fill_state_synthetic(cudaStream_t s, int n_pos, uint64_t seed) {
    RNB_TRY(reset(s));
    uint64_t id = seed * 131ull;
    auto cached = [&](void *p, size_t n) -> int {
        if (cfg.f32_math) return synth_dense<float>(s, (float *)p, n, ++id, 0.f, 1.f);
        return synth_dense<bf16>(s, (bf16 *)p, n, ++id, 0.f, 1.f);
    };
    for (LayerRun &r : runs_)
        for (size_t i = 0; i < r.m.size(); i++) {
            const rnb_b200_mixer_cfg &m = layers_[r.layer].mixers[i].c;
            const MixerState &st = r.m[i];
            if (m.mixer == RNB_B200_MIXER_LATENT_ATTENTION) RNB_TRY(cached(st.cache, (size_t)n_pos * latent_ld(m)));
            if (m.mixer == RNB_B200_MIXER_ATTENTION) {
                const size_t rows = (size_t)std::min(n_pos, attention_ring(m)) * m.kv_heads;
                RNB_TRY(cached(st.cache, rows * m.dim));
                RNB_TRY(cached(st.values, rows * m.vdim));
            }
            if (st.state && n_pos > 0) RNB_TRY(synth_dense<float>(s, st.state, (size_t)m.heads * m.dim * m.vdim, ++id, 0.f, 1.f));
            if (st.shift && n_pos > 0) RNB_TRY(synth_dense<float>(s, st.shift, (size_t)cfg.width, ++id, 0.f, 1.f));
            if (st.conv_ring && n_pos > 0)
                RNB_TRY(synth_dense<float>(s, st.conv_ring, (size_t)delta_ring_rows(m.conv) * (2 * m.kv_heads * m.dim + m.heads * m.vdim), ++id, 0.f, 1.f));
        }
    RNB_CU(cudaStreamSynchronize(s));
    return RNB_B200_OK;
}

// ---- scratch --------------------------------------------------------------------------------------
bool LayerStack::absorbed(const rnb_b200_mixer_cfg &m, int n) const {
    if (n <= SMALL || cfg.f32_math) return true;
    return !causal_attention_vcols(m.vdim) || causal_attention_smem(m.dim + m.rot_dim, m.vdim) > 227 * 1024;
}

int LayerStack::piece() const {
    int p = cfg.f32_math ? 512 : 4096;
    each_mixer([&](const StackLayer &, const StackMixer &M) {
        if (M.c.mixer == RNB_B200_MIXER_LATENT_ATTENTION && absorbed(M.c, SMALL + 1)) p = 512;
    });
    return p;
}

// Tokens per chunk: long chunks move less state, short ones give more CTAs.
static int linear_chunk(int tokens, int ctas_per_chunk) {
    if (tokens <= 96) return tokens;
    for (int c = 256; c > 64; c /= 2)
        if ((tokens + c - 1) / c * ctas_per_chunk >= 256) return c;
    return 64;
}
static bool linear_tiled(const rnb_b200_mixer_cfg &m) { return m.dim % 8 == 0 && m.vdim % 8 == 0 && m.dim <= 256; }
static int linear_tile_warps(int vdim) { return std::min((vdim + 15) / 16, 8); }
static bool delta_tiled(const rnb_b200_mixer_cfg &m) { return m.dim % 16 == 0 && m.vdim % 8 == 0 && m.dim <= 256; }
// Tile kernel of the delta rule: channel blocks it is instantiated for, groups of 16 value columns per CTA (few, so that the heads
// spread over the SMs), rows of the prepared tiles.
struct DeltaTileShape {
    int dt, cw, col_blocks, ld_qk, ld_val;
};
static DeltaTileShape delta_tile_shape(const rnb_b200_mixer_cfg &m) {
    DeltaTileShape s;
    const int cols = (m.vdim + 15) / 16;
    s.dt = m.dim <= 32 ? 2 : m.dim <= 64 ? 4 : m.dim <= 128 ? 8 : 16;
    s.cw = std::min(cols, 2);
    s.col_blocks = (cols + s.cw - 1) / s.cw;
    s.ld_qk = 16 * s.dt + 8;
    s.ld_val = 16 * s.cw + 8;
    return s;
}
// CTAs that work on one chunk of tokens
static int linear_ctas(const rnb_b200_mixer_cfg &m) { const int w = 16 * linear_tile_warps(m.vdim); return m.heads * ((m.vdim + w - 1) / w); }

int LayerStack::alloc_scratch(StackScratch &b, int cap) {
    for (void *p : b.allocs) cudaFree(p);
    b = StackScratch();
    const bool small = cap <= SMALL;
    const size_t T = (size_t)cap, D = (size_t)cfg.width, es = narrow(cap) ? 2 : 4;
    size_t proj[4] = {1, 1, 1, 1}, zw = 1, ww = 1, ow = 1, aw = 1, auxw[2] = {0, 0}, streams = 1, qfw = 0, partw = 0, st = 0, dc = 0, kn = 0, vx = 0, qn = 0, cqk = 0, cv = 0, rec = 0, th = 0;
    auto most = [](size_t &a, size_t b) { a = std::max(a, b); };
    for (const StackLayer &L : layers_) {
        if (!L.norm1) continue;   // uses another layer's weights: the same sizes
        most(aw, (size_t)std::max(L.out_cols, L.n_ff));
        for (size_t i = 0; i < L.mixers.size(); i++) {
            const StackMixer &M = L.mixers[i];
            const rnb_b200_mixer_cfg &m = M.c;
            const size_t hd = (size_t)m.heads * m.dim, hv = (size_t)m.heads * m.vdim;
            const bool linear = m.mixer == RNB_B200_MIXER_WKV || m.mixer == RNB_B200_MIXER_RETENTION || m.mixer == RNB_B200_MIXER_GLA;
            if (joined_rows(m)) {
                most(proj[i], (size_t)M.in_rows);
                most(auxw[i], (size_t)std::max(M.aux_rows, M.w1.rows));
            }
            if (m.mixer == RNB_B200_MIXER_LATENT_ATTENTION) {
                most(proj[0], (size_t)m.heads * (m.dim + m.rot_dim) * (absorbed(m, cap) && es == 2 ? 2 : 1));
                most(zw, (size_t)(m.kv_rank + m.rot_dim));
                if (absorbed(m, cap)) {
                    most(qfw, (size_t)m.heads * (m.kv_rank + m.rot_dim + 32));
                    most(partw, (size_t)m.heads * (small ? attend_chunks_ : 1) * latent_part_ld(m.kv_rank));
                } else {
                    most(kn, (size_t)cfg.max_ctx * hd);
                    most(vx, (size_t)cfg.max_ctx * hv);
                }
            } else if (m.mixer == RNB_B200_MIXER_ATTENTION) {
                if (small) most(partw, (size_t)m.heads * attention_chunks(m) * (m.vdim + 2));
                else most(qn, hd);
            } else {
                most(ow, hv);
                if (m.mixer == RNB_B200_MIXER_WKV || m.mixer == RNB_B200_MIXER_RETENTION)
                    for (size_t &p : proj) most(p, std::max(hd, hv));
                if (m.mixer == RNB_B200_MIXER_WKV) streams = 5, most(zw, (size_t)M.w1.rows);
                if (m.mixer == RNB_B200_MIXER_WKV || m.mixer == RNB_B200_MIXER_GLA) most(ww, hd), most(th, (size_t)M.w1.rows);
                if (m.mixer == RNB_B200_MIXER_DELTA && !small && es == 2 && delta_tiled(m)) {
                    const DeltaTileShape ts = delta_tile_shape(m);
                    most(cqk, (size_t)m.kv_heads * 32 * ts.ld_qk);
                    most(cv, (size_t)m.heads * ts.col_blocks * 16 * ts.ld_val);
                    most(rec, (size_t)m.heads * DR_REC);
                }
                if (!small && linear) {
                    size_t nc = 1;   // most chunks any token count up to cap can have
                    for (int t = 1; t <= cap; t++) {
                        const int c = linear_chunk(t, linear_ctas(m));
                        most(nc, (size_t)((t + c - 1) / c));
                    }
                    most(st, nc * hd * m.vdim);
                    most(dc, nc * hd);
                }
            }
        }
    }
    auto get = [&](void *pp, size_t bytes) -> int { return bytes ? alloc((void **)pp, bytes, &b.allocs) : RNB_B200_OK; };
    for (int i = 0; i < 2; i++) RNB_TRY(get(&b.x[i], T * D * 4));
    if (loops_) RNB_TRY(get(&b.emb, T * D * 4));
    RNB_TRY(get(&b.h, T * D * streams * es));
    for (int i = 0; i < 4; i++) RNB_TRY(get(&b.p[i], T * proj[i] * es));
    for (int i = 0; i < 2; i++) RNB_TRY(get(&b.aux[i], T * auxw[i] * 4));
    RNB_TRY(get(&b.y, T * D * 4));
    RNB_TRY(get(&b.z, T * zw * 4));
    if (!small) RNB_TRY(get(&b.w, T * ww * 4));
    RNB_TRY(get(&b.o, T * ow * 4));
    RNB_TRY(get(&b.act, T * aw * es));
    RNB_CU(cudaMemset(b.act, 0, T * aw * es));   // padding columns meet zero weights: they only have to be finite
    RNB_CU(cudaStreamSynchronize(nullptr));      // the decoder's stream does not wait for the default one
    RNB_TRY(get(&b.qn, T * qn * es));
    RNB_TRY(get(&b.cqk, (T + 15) / 16 * cqk * 2));
    RNB_TRY(get(&b.cv, (T + 15) / 16 * cv * 2));
    RNB_TRY(get(&b.rec, (T + 15) / 16 * rec));
    RNB_TRY(get(&b.qf, T * qfw * 4));
    RNB_TRY(get(&b.part, T * partw * 4));
    RNB_TRY(get(&b.starts, st * 4));
    RNB_TRY(get(&b.decays, dc * 4));
    if (!small && narrow(cap)) RNB_TRY(get(&b.th, T * th * 2 * 2));
    RNB_TRY(get(&b.kn, kn * 2));
    RNB_TRY(get(&b.vx, vx * 2));
    RNB_TRY(get(&b.rows, T * 4));
    RNB_TRY(get(&b.tok, T * 4));
    if (small) RNB_TRY(get(&b.logits, T * cfg.vocab * 4));
    b.cap = cap;
    return RNB_B200_OK;
}

int LayerStack::reserve(int tokens) {
    if (tokens <= SMALL || tokens <= big_.cap) return RNB_B200_OK;
    return alloc_scratch(big_, std::min(std::max(tokens, 256), piece()));
}

int LayerStack::ready(cudaStream_t s) {
    if (ready_) return RNB_B200_OK;
    for (Slot &t : slots_)
        if (!t.set) return fail(RNB_B200_VALIDATION_FAILED, "stack: tensor '%s' is not set", t.name.c_str());
    for (size_t i = 0; i < layers_.size(); i++)
        for (const StackMixer &M : layers_[i].mixers) {
            const bool gla = M.c.mixer == RNB_B200_MIXER_GLA;
            if (M.w1.rows != M.w2.cols) return fail(RNB_B200_VALIDATION_FAILED, "layer %zu: %s has %d rows, %s %d columns", i, gla ? "a1" : "w1", M.w1.rows, gla ? "a2" : "w2", M.w2.cols);
        }
    int optin = 0;
    RNB_CU(cudaDeviceGetAttribute(&optin, cudaDevAttrMaxSharedMemoryPerBlockOptin, state().device));
    auto raise = [&](const void *f) -> int {
        cudaFuncAttributes fa;
        RNB_CU(cudaFuncGetAttributes(&fa, f));
        RNB_CU(cudaFuncSetAttribute(f, cudaFuncAttributeMaxDynamicSharedMemorySize, optin - (int)fa.sharedSizeBytes));
        return RNB_B200_OK;
    };
    const void *fns[] = {(const void *)residual_norm_kernel<float, 4>, (const void *)residual_norm_kernel<float, 1>, (const void *)residual_norm_kernel<bf16, 4>,
                         (const void *)residual_norm_kernel<bf16, 1>, (const void *)dense_gemm_kernel, (const void *)decay_rows_kernel,
                         (const void *)linear_state_step_kernel<4>, (const void *)linear_state_step_kernel<8>, (const void *)linear_state_step_kernel<16>,
                         (const void *)linear_state_step_kernel<32>, (const void *)linear_state_step_kernel<64>, (const void *)causal_attention_kernel<4>,
                         (const void *)causal_attention_kernel<8>, (const void *)causal_attention_kernel<16>, (const void *)causal_attention_kernel<32>,
                         (const void *)attention_step_kernel<float, float>, (const void *)attention_step_kernel<float, bf16>, (const void *)attention_step_kernel<bf16, bf16>,
                         (const void *)delta_prepare_kernel<0>, (const void *)delta_prepare_kernel<2>,
                         (const void *)delta_prepare_kernel<3>, (const void *)delta_prepare_kernel<4>, (const void *)delta_tile_kernel<2>, (const void *)delta_tile_kernel<4>, (const void *)delta_tile_kernel<8>,
                         (const void *)delta_tile_kernel<16>};
    const void *pairs[] = {
#define RNB_AD(TI) (const void *)attention_delta_step_kernel<float, TI>, (const void *)attention_delta_step_kernel<bf16, TI>
        RNB_AD(4), RNB_AD(8), RNB_AD(16), RNB_AD(32), RNB_AD(64)
#undef RNB_AD
    };
    for (const void *f : pairs) RNB_TRY(raise(f));
    for (const void *f : fns) RNB_TRY(raise(f));
    const void *linear[] = {
#define RNB_LC(AT, MODE) (const void *)linear_state_chunk_kernel<AT, false, MODE>, (const void *)linear_state_chunk_kernel<AT, true, MODE>
#define RNB_LT(DT, MODE) (const void *)linear_state_tile_kernel<DT, false, MODE>, (const void *)linear_state_tile_kernel<DT, true, MODE>
#define RNB_LM(MODE) RNB_LC(float, MODE), RNB_LC(bf16, MODE), RNB_LT(2, MODE), RNB_LT(4, MODE), RNB_LT(8, MODE), RNB_LT(16, MODE)
        RNB_LM(LS_BONUS), RNB_LM(LS_HEAD_DECAY), RNB_LM(LS_UPDATED)
#undef RNB_LM
#undef RNB_LT
#undef RNB_LC
    };
    for (const void *f : linear) RNB_TRY(raise(f));
    const void *lat[] = {(const void *)latent_attend_mma_kernel<1>, (const void *)latent_attend_mma_kernel<2>, (const void *)latent_attend_mma_kernel<4>,
                         (const void *)latent_attend_mma_kernel<8>, (const void *)latent_attend_mma_kernel<10>, (const void *)latent_prepare_kernel<float, float>,
                         (const void *)latent_prepare_kernel<bf16, float>, (const void *)latent_prepare_kernel<bf16, bf16>, (const void *)latent_output_kernel<float>, (const void *)latent_output_kernel<bf16>};
    for (const void *f : lat) RNB_TRY(raise(f));
    for (StackLayer &L : layers_)
        for (StackMixer &M : L.mixers)
            if (M.w2.w && M.w2.cols % 4 == 0 && !cfg.f32_math) {
                DenseMat &m = M.w2x;
                const size_t pitch = (size_t)M.w2.cols * 2;
                RNB_TRY(alloc((void **)&m.w, (size_t)M.w2.rows * pitch * 2));
                for (int half = 0; half < 2; half++)
                    RNB_CU(cudaMemcpy2DAsync((char *)m.w + half * pitch, 2 * pitch, M.w2.w, pitch, pitch, (size_t)M.w2.rows, cudaMemcpyDeviceToDevice, s));
                m.rows = M.w2.rows;
                m.cols = 2 * M.w2.cols;
                m.tiled = true;
                PgTensorMap t;
                RNB_TRY(encode_token_map(&t, m.w, (size_t)m.rows, (size_t)m.cols, (size_t)m.cols, 64));
                memcpy(m.map, &t, sizeof(m.map));
            }
    RNB_TRY(alloc_scratch(small_, SMALL));
    RNB_TRY(reset(s));
    for (StackLayer &L : layers_)
        for (StackMixer &M : L.mixers)
            if (M.conv) {   // [channels][taps] as the tensors have them -> [taps][channels]
                const size_t taps = (size_t)M.c.conv, C = (size_t)2 * M.c.kv_heads * M.c.dim + (size_t)M.c.heads * M.c.vdim;
                std::vector<float> in(C * taps), out(C * taps);
                RNB_CU(cudaMemcpy(in.data(), M.conv, in.size() * 4, cudaMemcpyDeviceToHost));
                for (size_t c = 0; c < C; c++)
                    for (size_t t = 0; t < taps; t++) out[t * C + c] = in[c * taps + t];
                RNB_CU(cudaMemcpy(M.conv, out.data(), out.size() * 4, cudaMemcpyHostToDevice));
            }
    ready_ = true;
    return RNB_B200_OK;
}

int LayerStack::reset(cudaStream_t s) {
    // rings and caches hold nothing that position 0 could see
    for (LayerRun &r : runs_)
        for (size_t i = 0; i < r.m.size(); i++) {
            const rnb_b200_mixer_cfg &m = layers_[r.layer].mixers[i].c;
            if (r.m[i].state) RNB_CU(cudaMemsetAsync(r.m[i].state, 0, (size_t)m.heads * m.dim * m.vdim * 4, s));
            if (r.m[i].shift) RNB_CU(cudaMemsetAsync(r.m[i].shift, 0, (size_t)cfg.width * 4, s));
        }
    return RNB_B200_OK;
}

uint64_t LayerStack::cache_bytes_per_pos() const {
    uint64_t n = 0;
    for (const LayerRun &r : runs_)
        for (const StackMixer &M : layers_[r.layer].mixers) {
            const rnb_b200_mixer_cfg &m = M.c;
            const uint64_t row = m.mixer == RNB_B200_MIXER_LATENT_ATTENTION ? (uint64_t)latent_ld(m) : m.mixer == RNB_B200_MIXER_ATTENTION ? (uint64_t)m.kv_heads * (m.dim + m.vdim) : 0;
            n += row * (cfg.f32_math ? 4 : 2);
        }
    return n;
}

// ---- matrix products ------------------------------------------------------------------------------
int LayerStack::matmul(cudaStream_t s, int n, const Mm *jobs, int n_jobs, int *err) {
    if (n_jobs < 1 || n_jobs > DENSE_MAX_JOBS) return fail(RNB_B200_VALIDATION_FAILED, "stack: %d matrices in one launch", n_jobs);
    if (n <= SMALL) {
        DenseVecJobs J;
        memset(&J, 0, sizeof(J));
        J.n = n_jobs;
        int ctas = 0, all = 0, cols = 1 << 30;
        for (int i = 0; i < n_jobs; i++) {
            all += jobs[i].w2 ? jobs[i].w->rows : (jobs[i].w->rows + 1) / 2;
            cols = std::min(cols, jobs[i].w->cols);
        }
        // few rows: several warps share a pair of them, so that every SM has loads in flight to the end
        J.ksplit = all <= 4096 && cols >= 4096 ? 4 : all <= 12288 && cols >= 2048 ? 2 : 1;
        const int per_cta = DV_WARPS / J.ksplit;
        for (int i = 0; i < n_jobs; i++) {
            DenseVecJob &j = J.j[i];
            j.w = reinterpret_cast<const bf16 *>(jobs[i].w->w);
            j.w2 = jobs[i].w2 ? reinterpret_cast<const bf16 *>(jobs[i].w2->w) : nullptr;
            j.x = reinterpret_cast<const float *>(jobs[i].x);
            j.y = reinterpret_cast<float *>(jobs[i].y);
            j.rows = jobs[i].w->rows;
            j.cols = jobs[i].w->cols;
            j.ldx = (int)jobs[i].ldx;
            j.ldy = (int)(jobs[i].ldy ? jobs[i].ldy : (size_t)j.rows);
            j.act = cfg.act;
            j.cta0 = ctas;
            j.vec = jobs[i].w->cols % 8 == 0 && ((uintptr_t)j.x & 15) == 0 && j.ldx % 4 == 0;
            const int units = j.w2 ? j.rows : (j.rows + 1) / 2;
            ctas += (units + per_cta - 1) / per_cta;
        }
        const dim3 grid((unsigned)ctas), block(DV_WARPS * 32);
        if (n == 1) RNB_CU(launch_k(dense_gemv_kernel<1>, grid, block, 0, s, J));
        else if (n == 2) RNB_CU(launch_k(dense_gemv_kernel<2>, grid, block, 0, s, J));
        else if (n <= 4) RNB_CU(launch_k(dense_gemv_kernel<4>, grid, block, 0, s, J));
        else RNB_CU(launch_k(dense_gemv_kernel<8>, grid, block, 0, s, J));
        return RNB_B200_OK;
    }
    bool tiled = !cfg.f32_math;
    for (int i = 0; i < n_jobs; i++) tiled = tiled && jobs[i].w->tiled && (!jobs[i].w2 || jobs[i].w2->tiled) && jobs[i].ldx % 8 == 0 && ((uintptr_t)jobs[i].x & 15) == 0;
    if (tiled) {
        DenseGemmJobs J;
        DenseMaps M;
        memset(&J, 0, sizeof(J));
        memset(&M, 0, sizeof(M));
        J.n = n_jobs;
        J.seq = n;
        int tiles = 0;
        for (int i = 0; i < n_jobs; i++) {
            DenseGemmJob &j = J.j[i];
            j.y = jobs[i].y;
            j.decay_bias = jobs[i].decay_bias;
            if (jobs[i].decay && jobs[i].decay->mixer == RNB_B200_MIXER_GLA) j.decay_kind = DECAY_SIGMOID_ROOT, j.inv_tau = 1.0f / jobs[i].decay->tau;
            j.act = cfg.act;
            j.rows = jobs[i].w->rows;
            j.ld = (int)(jobs[i].ldy ? jobs[i].ldy : (size_t)j.rows);
            j.cols = jobs[i].w->cols;
            j.tile0 = tiles;
            j.out_bf16 = !jobs[i].f32_out;
            j.pair = jobs[i].w2 != nullptr;
            const int per = j.pair ? DG_ROWS / 2 : DG_ROWS;
            tiles += (j.rows + per - 1) / per;
            RNB_TRY(encode_token_map(&M.x[i], reinterpret_cast<const uint16_t *>(jobs[i].x), (size_t)n, (size_t)j.cols, jobs[i].ldx, DG_TOK));
            memcpy(&M.w[i], jobs[i].w->map, sizeof(PgTensorMap));
            if (j.pair) memcpy(&M.w2[i], jobs[i].w2->map, sizeof(PgTensorMap));
        }
        RNB_CU(launch_k(dense_gemm_kernel, dim3((unsigned)((n + DG_TOK - 1) / DG_TOK), (unsigned)tiles), dim3(DG_THREADS), DG_SMEM, s, J, M, err));
        return RNB_B200_OK;
    }
    DenseSimtJobs J;
    memset(&J, 0, sizeof(J));
    J.n = n_jobs;
    J.seq = n;
    int tiles = 0;
    for (int i = 0; i < n_jobs; i++) {
        DenseSimtJob &j = J.j[i];
        j.w = reinterpret_cast<const bf16 *>(jobs[i].w->w);
        j.w2 = jobs[i].w2 ? reinterpret_cast<const bf16 *>(jobs[i].w2->w) : nullptr;
        j.x = jobs[i].x;
        j.y = jobs[i].y;
        j.rows = jobs[i].w->rows;
        j.ld = (int)(jobs[i].ldy ? jobs[i].ldy : (size_t)j.rows);
        j.act = cfg.act;
        j.cols = jobs[i].w->cols;
        j.ldx = (int)jobs[i].ldx;
        j.tile0 = tiles;
        j.out_bf16 = !jobs[i].f32_out && !cfg.f32_math;
        tiles += (j.rows + DS_TILE - 1) / DS_TILE;
    }
    const dim3 grid((unsigned)tiles, (unsigned)((n + DS_TILE - 1) / DS_TILE));
    if (cfg.f32_math) RNB_CU(launch_k(dense_gemm_simt_kernel<float>, grid, dim3(256), 0, s, J));
    else RNB_CU(launch_k(dense_gemm_simt_kernel<bf16>, grid, dim3(256), 0, s, J));
    return RNB_B200_OK;
}

// ---- one step -------------------------------------------------------------------------------------
// residual_norm_kernel with the row buffers of `b`; `cur` is the buffer that holds the residual.
int LayerStack::boundary(cudaStream_t s, int n, StackScratch &b, int &cur, const float *y, const float *wb, bool emb, const float *wn, const float *bn, const StackLayer *shift, LayerRun *run) {
    ResidualNormArgs a;
    memset(&a, 0, sizeof(a));
    a.x_in = a.x_out = b.x[cur];
    a.y = y;
    a.wb = wb;
    a.emb = emb ? b.emb : nullptr;
    a.wn = wn;
    a.bn = bn;
    a.center = cfg.norm == RNB_B200_NORM_LAYER;
    a.h = b.h;
    a.mult = cfg.residual_mult;
    a.eps = cfg.norm_eps;
    a.width = cfg.width;
    a.tokens = n;
    a.rows_per_cta = shift ? 8 : 1;
    if (shift) {
        a.mu = shift->mixers[0].mu;
        a.n_mix = 5;
        a.shift_in = run->m[0].shift;
        a.shift_out = n <= a.rows_per_cta ? run->m[0].shift : run->m[0].shift_out;
        if (n > a.rows_per_cta && (y || emb)) {
            // a CTA recomputes the row before its first from the old residual: the new one needs its own buffer
            a.x_out = b.x[cur ^ 1];
            cur ^= 1;
        }
    }
    const bool v4 = cfg.width % 4 == 0;
    const int per = v4 ? 4 : 1, want = (cfg.width + per - 1) / per;
    const int threads = std::max(32, std::min(n <= SMALL ? 1024 : 512, (want + 31) / 32 * 32));
    const size_t smem = (size_t)cfg.width * 4 * (shift ? 2 : 1);
    const dim3 grid((unsigned)((n + a.rows_per_cta - 1) / a.rows_per_cta)), block((unsigned)threads);
    if (narrow(n)) {
        if (v4) RNB_CU(launch_k(residual_norm_kernel<bf16, 4>, grid, block, smem, s, a));
        else RNB_CU(launch_k(residual_norm_kernel<bf16, 1>, grid, block, smem, s, a));
    } else {
        if (v4) RNB_CU(launch_k(residual_norm_kernel<float, 4>, grid, block, smem, s, a));
        else RNB_CU(launch_k(residual_norm_kernel<float, 1>, grid, block, smem, s, a));
    }
    if (shift && a.shift_out != a.shift_in) RNB_CU(cudaMemcpyAsync(run->m[0].shift, run->m[0].shift_out, (size_t)cfg.width * 4, cudaMemcpyDeviceToDevice, s));
    return RNB_B200_OK;
}

// linear_state_scan_kernel between the two passes over the chunks
static int launch_linear_scan(cudaStream_t s, const LinearChunkArgs &a) {
    const size_t n = (size_t)a.heads * a.dim * a.vdim;
    const float *decays = a.w ? a.decays : nullptr;
    if (a.vdim % 4 == 0) RNB_CU(launch_k(linear_state_scan_kernel<4>, dim3((unsigned)((n / 4 + 255) / 256)), dim3(256), 0, s, (const float *)a.state, a.starts, decays, a.decay, a.heads, a.dim, a.vdim, a.chunk, a.n_chunks));
    else RNB_CU(launch_k(linear_state_scan_kernel<1>, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, s, (const float *)a.state, a.starts, decays, a.decay, a.heads, a.dim, a.vdim, a.chunk, a.n_chunks));
    return RNB_B200_OK;
}
template <int DT, int MODE>
static int launch_linear_tiles(cudaStream_t s, const LinearChunkArgs &a) {
    const int nw = linear_tile_warps(a.vdim);
    const unsigned zb = (unsigned)((a.vdim + 16 * nw - 1) / (16 * nw));
    const size_t smem = linear_tile_smem(DT, nw).bytes;
    const dim3 block((unsigned)(32 * nw));
    if (a.n_chunks > 1) {
        RNB_CU(launch_k(linear_state_tile_kernel<DT, false, MODE>, dim3((unsigned)(a.n_chunks - 1), (unsigned)a.heads, zb), block, smem, s, a));
        RNB_TRY(launch_linear_scan(s, a));
    }
    RNB_CU(launch_k(linear_state_tile_kernel<DT, true, MODE>, dim3((unsigned)a.n_chunks, (unsigned)a.heads, zb), block, smem, s, a));
    return RNB_B200_OK;
}
template <class AT, int MODE>
static int launch_linear_chunks(cudaStream_t s, LinearChunkArgs a) {
    a.G = round_pow2((a.dim + LS_TI - 1) / LS_TI);
    a.JG = std::min((a.vdim + 3) / 4, 256 / a.G);
    const dim3 block((unsigned)((a.G * a.JG + 31) / 32 * 32));
    const unsigned zb = (unsigned)((a.vdim + 4 * a.JG - 1) / (4 * a.JG));
    const size_t smem = linear_chunk_smem(a.G, a.JG);
    if (a.n_chunks > 1) {
        RNB_CU(launch_k(linear_state_chunk_kernel<AT, false, MODE>, dim3((unsigned)(a.n_chunks - 1), (unsigned)a.heads, zb), block, smem, s, a));
        RNB_TRY(launch_linear_scan(s, a));
    }
    RNB_CU(launch_k(linear_state_chunk_kernel<AT, true, MODE>, dim3((unsigned)a.n_chunks, (unsigned)a.heads, zb), block, smem, s, a));
    return RNB_B200_OK;
}
template <int MODE>
static int launch_linear(cudaStream_t s, const LinearChunkArgs &a, bool narrow, bool tiled) {
    if (!narrow) return launch_linear_chunks<float, MODE>(s, a);
    if (!tiled) return launch_linear_chunks<bf16, MODE>(s, a);
    if (a.dim <= 32) return launch_linear_tiles<2, MODE>(s, a);
    if (a.dim <= 64) return launch_linear_tiles<4, MODE>(s, a);
    if (a.dim <= 128) return launch_linear_tiles<8, MODE>(s, a);
    return launch_linear_tiles<16, MODE>(s, a);
}

static int launch_causal_attention(cudaStream_t s, const CausalAttentionArgs &a);

// Norm and gate of a mixer's heads in b.o; the result is its part of the output matrix's input.
int LayerStack::head_norm_gate(cudaStream_t s, int n, StackScratch &b, const StackLayer &L, const StackMixer &M, const void *g, int ldg) {
    HeadNormGateArgs a;
    memset(&a, 0, sizeof(a));
    a.o = b.o, a.w = M.head_norm, a.g = g, a.act = act_of(b, M, n);
    a.eps = cfg.norm_eps, a.mul = M.c.out_scale;
    a.heads = M.c.heads, a.vdim = M.c.vdim;
    a.w_head = M.c.mixer == RNB_B200_MIXER_WKV ? M.c.vdim : 0;
    a.ldg = ldg, a.lda = L.out_cols;
    const int v = a.vdim % 4 == 0 && ldg % 4 == 0 ? 4 : 1;
    a.lanes = std::min(32, round_pow2((a.vdim + v - 1) / v));
    a.units = (size_t)n * a.heads;
    const dim3 grid((unsigned)((a.units * a.lanes + 255) / 256));
    if (narrow(n)) {
        if (v == 4) RNB_CU(launch_k(head_norm_gate_kernel<bf16, 4>, grid, dim3(256), 0, s, a));
        else RNB_CU(launch_k(head_norm_gate_kernel<bf16, 1>, grid, dim3(256), 0, s, a));
    } else {
        if (v == 4) RNB_CU(launch_k(head_norm_gate_kernel<float, 4>, grid, dim3(256), 0, s, a));
        else RNB_CU(launch_k(head_norm_gate_kernel<float, 1>, grid, dim3(256), 0, s, a));
    }
    return RNB_B200_OK;
}

// Time mixing, retention, gated linear attention: recurrence, head norm and gate behind the projections.
int LayerStack::mixer_linear(cudaStream_t s, int n, StackScratch &b, StackLayer &L, int i, MixerState &R, const int *pos_dev, int *err) {
    const StackMixer &M = L.mixers[i];
    const rnb_b200_mixer_cfg &m = M.c;
    const int mode = m.mixer == RNB_B200_MIXER_WKV ? LS_BONUS : m.mixer == RNB_B200_MIXER_RETENTION ? LS_HEAD_DECAY : LS_UPDATED;
    const bool nb = narrow(n), gla = mode == LS_UPDATED;
    const Rotation rot{(const float2 *)M.rot_table, m.rot.dims, m.rot.interleaved};
    const float k_mul = mode == LS_HEAD_DECAY ? 1.f / sqrtf((float)m.dim) : 1.f, o_mul = gla ? 1.f / sqrtf((float)m.dim) : 1.f;
    auto part = [&](int j) -> void * { return gla ? (void *)((char *)b.p[i] + (size_t)M.in_at[j] * (nb ? 2 : 4)) : b.p[j]; };
    float *z = gla ? b.aux[i] : b.z;
    const int ldr = gla ? M.in_rows : m.heads * m.dim, ldv = gla ? M.in_rows : m.heads * m.vdim, rank = M.w1.rows;
    if (n <= SMALL) {
        LinearStepArgs a;
        memset(&a, 0, sizeof(a));
        a.r = (const float *)part(0), a.k = (const float *)part(1), a.v = (const float *)part(2), a.g = (const float *)part(3);
        a.z = z, a.w0 = M.w0, a.decay = M.decay, a.u = M.u;
        a.w2 = reinterpret_cast<const bf16 *>(M.w2.w);
        a.norm = M.head_norm, a.norm_head = gla ? 0 : m.vdim;
        a.rot = rot;
        a.pos0 = pos_dev;
        a.k_mul = k_mul, a.o_mul = o_mul, a.out_mul = m.out_scale, a.eps = cfg.norm_eps;
        a.inv_tau = gla ? 1.f / m.tau : 0.f;
        a.state = R.state, a.o = b.o, a.act = (float *)act_of(b, M, n);
        a.counters = counters_ + i * counters_of_mixer_;
        a.tokens = n, a.heads = m.heads, a.dim = m.dim, a.vdim = m.vdim, a.rank = rank, a.mode = mode;
        a.ldr = ldr, a.ldv = ldv, a.lda = L.out_cols;
        const dim3 grid((unsigned)m.heads, (unsigned)((m.vdim + 31) / 32)), block(256);
        const size_t smem = linear_step_smem(n, m.dim, a.rank);
        const int ti = (m.dim + 7) / 8;
        if (ti <= 4) RNB_CU(launch_k(linear_state_step_kernel<4>, grid, block, smem, s, a));
        else if (ti <= 8) RNB_CU(launch_k(linear_state_step_kernel<8>, grid, block, smem, s, a));
        else if (ti <= 16) RNB_CU(launch_k(linear_state_step_kernel<16>, grid, block, smem, s, a));
        else if (ti <= 32) RNB_CU(launch_k(linear_state_step_kernel<32>, grid, block, smem, s, a));
        else RNB_CU(launch_k(linear_state_step_kernel<64>, grid, block, smem, s, a));
        return RNB_B200_OK;
    }
    if (mode != LS_HEAD_DECAY) {
        const int ch = m.heads * m.dim, kind = gla ? DECAY_SIGMOID_ROOT : DECAY_EXP;
        if (nb && M.w2x.w) {
            const size_t nz = (size_t)n * rank;
            RNB_CU(launch_k(split_rows_kernel, dim3((unsigned)((nz + 255) / 256)), dim3(256), 0, s, (const float *)z, rank, nz, kind, reinterpret_cast<bf16 *>(b.th)));
            const Mm dj = {&M.w2x, nullptr, b.th, (size_t)2 * rank, b.w, true, 0, M.w0, &m};
            RNB_TRY(matmul(s, n, &dj, 1, err));
        } else
            RNB_CU(launch_k(decay_rows_kernel, dim3((unsigned)((ch + 127) / 128), (unsigned)((n + 15) / 16)), dim3(128), (size_t)rank * 64, s, (const float *)z,
                        reinterpret_cast<const bf16 *>(M.w2.w), (const float *)M.w0, n, rank, ch, kind, gla ? 1.f / m.tau : 0.f, b.w));
    } else {
        RotateArgs r;
        memset(&r, 0, sizeof(r));
        r.x[0] = b.p[0], r.x[1] = b.p[1];
        r.mul[0] = 1.f, r.mul[1] = k_mul;
        r.heads = m.heads, r.hd = m.dim;
        r.rot = rot;
        r.pos0 = pos_dev;
        if (nb) RNB_CU(launch_k(rotate_heads_kernel<bf16>, dim3((unsigned)n, 2), dim3(256), 0, s, r));
        else RNB_CU(launch_k(rotate_heads_kernel<float>, dim3((unsigned)n, 2), dim3(256), 0, s, r));
    }
    LinearChunkArgs a;
    memset(&a, 0, sizeof(a));
    a.r = part(0), a.k = part(1), a.v = part(2);
    a.w = mode == LS_HEAD_DECAY ? nullptr : b.w;
    a.decay = M.decay, a.u = M.u, a.o_mul = o_mul;
    a.state = R.state, a.o = b.o, a.starts = b.starts, a.decays = b.decays;
    a.tokens = n, a.heads = m.heads, a.dim = m.dim, a.vdim = m.vdim, a.ldr = ldr, a.ldv = ldv;
    a.chunk = linear_chunk(n, linear_ctas(m));
    a.n_chunks = (n + a.chunk - 1) / a.chunk;
    if (mode == LS_BONUS) RNB_TRY(launch_linear<LS_BONUS>(s, a, nb, linear_tiled(m)));
    else if (mode == LS_HEAD_DECAY) RNB_TRY(launch_linear<LS_HEAD_DECAY>(s, a, nb, linear_tiled(m)));
    else RNB_TRY(launch_linear<LS_UPDATED>(s, a, nb, linear_tiled(m)));
    return head_norm_gate(s, n, b, L, M, part(3), ldv);
}

WindowAttentionArgs LayerStack::attention_args(int n, StackScratch &b, StackLayer &L, int i, MixerState &R, const int *pos_dev) const {
    const StackMixer &M = L.mixers[i];
    const rnb_b200_mixer_cfg &m = M.c;
    const bool nb = narrow(n);
    const char *p = (const char *)b.p[i];
    const size_t es = nb ? 2 : 4;
    WindowAttentionArgs a;
    memset(&a, 0, sizeof(a));
    a.q = p, a.k = p + M.in_at[1] * es, a.v = p + M.in_at[2] * es;
    a.qn = b.qn, a.kc = R.cache, a.vc = R.values;
    a.gate = m.head_gate ? b.aux[i] : nullptr, a.ldg = M.aux_rows;
    a.part = b.part, a.counters = counters_ + i * counters_of_mixer_, a.act = act_of(b, M, n);
    a.fresh = n <= SMALL;
    a.pos0 = pos_dev;
    a.rot = Rotation{(const float2 *)M.rot_table, m.rot.dims, m.rot.interleaved};
    a.eps = cfg.norm_eps, a.scale = m.scale, a.out_mul = m.out_scale;
    a.tokens = n, a.heads = m.heads, a.kv_heads = m.kv_heads, a.dim = m.dim, a.vdim = m.vdim, a.ld = M.in_rows, a.lda = L.out_cols;
    a.ring = attention_ring(m), a.window = m.window, a.qk_norm = m.qk_norm;
    a.fours = m.dim % 4 == 0 && m.rot.dims % 4 == 0 && (m.rot.interleaved || !a.rot.table);
    return a;
}

int LayerStack::mixer_attention(cudaStream_t s, int n, StackScratch &b, StackLayer &L, int i, MixerState &R, const int *pos_dev) {
    const rnb_b200_mixer_cfg &m = L.mixers[i].c;
    const bool nb = narrow(n);
    const WindowAttentionArgs a = attention_args(n, b, L, i, R, pos_dev);
    const size_t smem = attention_step_bytes(m, cfg.f32_math != 0);
    if (n <= SMALL) {
        const dim3 grid((unsigned)attention_chunks(m), (unsigned)m.kv_heads, (unsigned)n);
        if (cfg.f32_math) RNB_CU(launch_k(attention_step_kernel<float, float>, grid, dim3(AS_THREADS), smem, s, a));
        else RNB_CU(launch_k(attention_step_kernel<float, bf16>, grid, dim3(AS_THREADS), smem, s, a));
        return RNB_B200_OK;
    }
    const dim3 pg((unsigned)n, (unsigned)((m.heads + 2 * m.kv_heads + 7) / 8)), one(1, (unsigned)m.kv_heads, (unsigned)n);
    if (!nb) {
        RNB_CU(launch_k(attention_prepare_kernel<float, float>, pg, dim3(256), 0, s, a));
        RNB_CU(launch_k(attention_step_kernel<float, float>, one, dim3(AS_THREADS), smem, s, a));
        return RNB_B200_OK;
    }
    RNB_CU(launch_k(attention_prepare_kernel<bf16, bf16>, pg, dim3(256), 0, s, a));
    if (!attention_tiled(m)) {
        RNB_CU(launch_k(attention_step_kernel<bf16, bf16>, one, dim3(AS_THREADS), smem, s, a));
        return RNB_B200_OK;
    }
    CausalAttentionArgs c;
    memset(&c, 0, sizeof(c));
    c.q = (const bf16 *)b.qn, c.k = (const bf16 *)R.cache, c.v = (const bf16 *)R.values;
    c.act = (bf16 *)a.act, c.gate = a.gate, c.pos0 = pos_dev;
    c.ldq = (size_t)m.heads * m.dim, c.ldk = (size_t)m.kv_heads * m.dim, c.ldv = (size_t)m.kv_heads * m.vdim;
    c.scale = m.scale, c.out_mul = m.out_scale;
    c.tokens = n, c.heads = m.heads, c.group = m.heads / m.kv_heads, c.dim = m.dim, c.vdim = m.vdim;
    c.ring = a.ring, c.window = m.window, c.lda = a.lda, c.ldg = a.ldg;
    c.vec = m.dim % 8 == 0 && m.vdim % 8 == 0;
    return launch_causal_attention(s, c);
}

DeltaArgs LayerStack::delta_args(int n, StackScratch &b, StackLayer &L, int i, MixerState &R, const int *pos_dev) const {
    const StackMixer &M = L.mixers[i];
    const rnb_b200_mixer_cfg &m = M.c;
    DeltaArgs a;
    memset(&a, 0, sizeof(a));
    a.p = b.p[i], a.ba = b.aux[i], a.conv = M.conv, a.a_log = M.a_log, a.dt = M.dt, a.norm = M.head_norm;
    a.ring = R.conv_ring, a.state = R.state, a.o = b.o, a.counters = counters_ + i * counters_of_mixer_, a.pos0 = pos_dev;
    if (n <= SMALL) a.act = (float *)act_of(b, M, n);
    const DeltaTileShape ts = delta_tile_shape(m);
    a.cqk = reinterpret_cast<bf16 *>(b.cqk), a.cv = reinterpret_cast<bf16 *>(b.cv), a.rec = b.rec;
    a.ld_qk = ts.ld_qk, a.ld_val = ts.ld_val, a.col_blocks = ts.col_blocks, a.cw = ts.cw;
    a.eps = cfg.norm_eps, a.out_mul = m.out_scale, a.q_mul = 1.0f / sqrtf((float)m.dim);
    a.tokens = n, a.heads = m.heads, a.kv_heads = m.kv_heads, a.dim = m.dim, a.vdim = m.vdim, a.taps = m.conv;
    a.k_at = M.in_at[1], a.v_at = M.in_at[2], a.g_at = M.in_at[3], a.a_at = m.heads, a.ld = M.in_rows, a.ld_ba = M.aux_rows, a.lda = L.out_cols;
    return a;
}

int LayerStack::mixer_delta(cudaStream_t s, int n, StackScratch &b, StackLayer &L, int i, MixerState &R, const int *pos_dev, int *err) {
    const StackMixer &M = L.mixers[i];
    const rnb_b200_mixer_cfg &m = M.c;
    const bool nb = narrow(n);
    DeltaArgs a = delta_args(n, b, L, i, R, pos_dev);
    a.err = err;
    if (nb && delta_tiled(m)) {
        const dim3 pg((unsigned)((n + DP_TOKENS - 1) / DP_TOKENS), (unsigned)m.kv_heads);
        const size_t psmem = delta_prepare_smem(m.dim);
        if (m.conv == 2) RNB_CU(launch_k(delta_prepare_kernel<2>, pg, dim3(256), psmem, s, a));
        else if (m.conv == 3) RNB_CU(launch_k(delta_prepare_kernel<3>, pg, dim3(256), psmem, s, a));
        else if (m.conv == 4) RNB_CU(launch_k(delta_prepare_kernel<4>, pg, dim3(256), psmem, s, a));
        else RNB_CU(launch_k(delta_prepare_kernel<0>, pg, dim3(256), psmem, s, a));
        const dim3 grid((unsigned)m.heads, (unsigned)a.col_blocks), block((unsigned)(32 * (DT_SPLIT * a.cw + 1)));
        const int dt = delta_tile_shape(m).dt;
        const size_t smem = delta_tile_smem(dt, a.cw).bytes;
        if (dt == 2) RNB_CU(launch_k(delta_tile_kernel<2>, grid, block, smem, s, a));
        else if (dt == 4) RNB_CU(launch_k(delta_tile_kernel<4>, grid, block, smem, s, a));
        else if (dt == 8) RNB_CU(launch_k(delta_tile_kernel<8>, grid, block, smem, s, a));
        else RNB_CU(launch_k(delta_tile_kernel<16>, grid, block, smem, s, a));
    } else {
        const dim3 grid((unsigned)m.heads, (unsigned)((m.vdim + 31) / 32)), block(256);
        const size_t smem = delta_step_smem(m.dim);
        const int ti = (m.dim + 7) / 8;
#define RNB_DS(TI) RNB_CU(nb ? launch_k(delta_step_kernel<bf16, TI>, grid, block, smem, s, a) : launch_k(delta_step_kernel<float, TI>, grid, block, smem, s, a))
        if (ti <= 4) RNB_DS(4);
        else if (ti <= 8) RNB_DS(8);
        else if (ti <= 16) RNB_DS(16);
        else if (ti <= 32) RNB_DS(32);
        else RNB_DS(64);
#undef RNB_DS
        if (n <= SMALL) return RNB_B200_OK;
        const dim3 rg((unsigned)((2 * m.kv_heads * m.dim + m.heads * m.vdim + 255) / 256));
        if (nb) RNB_CU(launch_k(delta_ring_kernel<bf16>, rg, dim3(256), 0, s, a));
        else RNB_CU(launch_k(delta_ring_kernel<float>, rg, dim3(256), 0, s, a));
    }
    return head_norm_gate(s, n, b, L, M, (const char *)b.p[i] + (size_t)a.g_at * (nb ? 2 : 4), M.in_rows);
}

static int launch_causal_attention(cudaStream_t s, const CausalAttentionArgs &a) {
    const dim3 grid((unsigned)((a.tokens + CA_ROWS - 1) / CA_ROWS), (unsigned)a.heads), block(CA_THREADS);
    const size_t smem = causal_attention_smem(a.dim + a.dim2, a.vdim);
    switch (causal_attention_vcols(a.vdim)) {
    case 32: RNB_CU(launch_k(causal_attention_kernel<4>, grid, block, smem, s, a)); break;
    case 64: RNB_CU(launch_k(causal_attention_kernel<8>, grid, block, smem, s, a)); break;
    case 128: RNB_CU(launch_k(causal_attention_kernel<16>, grid, block, smem, s, a)); break;
    default: RNB_CU(launch_k(causal_attention_kernel<32>, grid, block, smem, s, a));
    }
    return RNB_B200_OK;
}
// A few tokens of window attention and the delta rule side by side: one launch.
int LayerStack::mixers_attention_delta(cudaStream_t s, int n, StackScratch &b, StackLayer &L, LayerRun &R, const int *pos_dev) {
    const rnb_b200_mixer_cfg &m = L.mixers[0].c, &k = L.mixers[1].c;
    const WindowAttentionArgs a = attention_args(n, b, L, 0, R.m[0], pos_dev);
    const DeltaArgs d = delta_args(n, b, L, 1, R.m[1], pos_dev);
    const int chunks = attention_chunks(m), n_att = chunks * m.kv_heads * n, n_jb = (k.vdim + 31) / 32, ti = (k.dim + 7) / 8;
    const dim3 grid((unsigned)(n_att + k.heads * n_jb));
    const size_t smem = std::max(attention_step_bytes(m, cfg.f32_math != 0), delta_step_smem(k.dim));
#define RNB_AD(TI) RNB_CU(cfg.f32_math ? launch_k(attention_delta_step_kernel<float, TI>, grid, dim3(256), smem, s, a, d, chunks, n_att, n_jb) \
                                       : launch_k(attention_delta_step_kernel<bf16, TI>, grid, dim3(256), smem, s, a, d, chunks, n_att, n_jb))
    if (ti <= 4) RNB_AD(4);
    else if (ti <= 8) RNB_AD(8);
    else if (ti <= 16) RNB_AD(16);
    else if (ti <= 32) RNB_AD(32);
    else RNB_AD(64);
#undef RNB_AD
    return RNB_B200_OK;
}

static bool latent_mma_fits(const LatentDims &d) { return d.rank % 8 == 0 && d.rank <= 640 && latent_mma_smem(d).bytes <= 220 * 1024; }
static int launch_latent_attend_mma(cudaStream_t s, const bf16 *qf, const bf16 *cache, const LatentDims &d, float scale, const int *pos, float *part, int n, int chunks) {
    const dim3 grid((unsigned)chunks, (unsigned)((d.heads + 15) / 16), (unsigned)n), block(LM_THREADS);
    const size_t smem = latent_mma_smem(d).bytes;
    const int nt = (d.rank + 63) / 64;
    if (nt <= 1) RNB_CU(launch_k(latent_attend_mma_kernel<1>, grid, block, smem, s, qf, cache, d, scale, pos, part));
    else if (nt <= 2) RNB_CU(launch_k(latent_attend_mma_kernel<2>, grid, block, smem, s, qf, cache, d, scale, pos, part));
    else if (nt <= 4) RNB_CU(launch_k(latent_attend_mma_kernel<4>, grid, block, smem, s, qf, cache, d, scale, pos, part));
    else if (nt <= 8) RNB_CU(launch_k(latent_attend_mma_kernel<8>, grid, block, smem, s, qf, cache, d, scale, pos, part));
    else RNB_CU(launch_k(latent_attend_mma_kernel<10>, grid, block, smem, s, qf, cache, d, scale, pos, part));
    return RNB_B200_OK;
}
template <class CT>
static int launch_latent_attend(cudaStream_t s, const float *qf, const CT *cache, const LatentDims &d, float scale, const int *pos, float *part, int n, int chunks) {
    const dim3 grid((unsigned)chunks, (unsigned)d.heads, (unsigned)n), block(128);
    const int nq = (d.rank + d.rot_dim + 31) / 32;
    if (nq <= 2) RNB_CU(launch_k(latent_attend_kernel<CT, 2>, grid, block, 0, s, qf, cache, d, scale, pos, part));
    else if (nq <= 5) RNB_CU(launch_k(latent_attend_kernel<CT, 5>, grid, block, 0, s, qf, cache, d, scale, pos, part));
    else if (nq <= 10) RNB_CU(launch_k(latent_attend_kernel<CT, 10>, grid, block, 0, s, qf, cache, d, scale, pos, part));
    else if (nq <= 18) RNB_CU(launch_k(latent_attend_kernel<CT, 18>, grid, block, 0, s, qf, cache, d, scale, pos, part));
    else RNB_CU(launch_k(latent_attend_kernel<CT, 36>, grid, block, 0, s, qf, cache, d, scale, pos, part));
    return RNB_B200_OK;
}

int LayerStack::mixer_latent(cudaStream_t s, int n, StackScratch &b, StackLayer &L, int i, MixerState &R, const int *pos_dev, int pos_host, int *err) {
    const StackMixer &M = L.mixers[i];
    const rnb_b200_mixer_cfg &m = M.c;
    const LatentDims d{m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, latent_ld(m)};
    const Rotation rot{(const float2 *)M.rot_table, m.rot.dims, m.rot.interleaved};
    const bool ab = absorbed(m, n), nb = narrow(n);
    if (ab) {
        LatentPrepareArgs a;
        memset(&a, 0, sizeof(a));
        a.q = (const float *)b.p[0], a.y = b.z, a.w = M.dkv_norm;
        a.uk = reinterpret_cast<const bf16 *>(M.uk.w);
        const bool mma = !cfg.f32_math && latent_mma_fits(d);
        a.qf = b.qf, a.qld = mma ? (m.kv_rank + m.rot_dim + 31) & ~31 : m.kv_rank + m.rot_dim, a.cache = R.cache, a.pos0 = pos_dev, a.eps = cfg.norm_eps, a.d = d, a.rot = rot;
        const dim3 grid((unsigned)(m.heads + 1), (unsigned)n, (unsigned)((m.kv_rank + LP_COLS - 1) / LP_COLS)), pb(LP_THREADS);
        const size_t psmem = ((size_t)((m.dim + 3) & ~3) + LP_GROUPS * LP_COLS) * 4;
        const int chunks = n <= SMALL ? attend_chunks_ : 1;
        if (cfg.f32_math) {
            RNB_CU(launch_k(latent_prepare_kernel<float, float>, grid, pb, psmem, s, a));
            RNB_TRY(launch_latent_attend<float>(s, b.qf, (const float *)R.cache, d, m.scale, pos_dev, b.part, n, chunks));
        } else {
            if (mma) RNB_CU(launch_k(latent_prepare_kernel<bf16, bf16>, grid, pb, psmem, s, a));
            else RNB_CU(launch_k(latent_prepare_kernel<bf16, float>, grid, pb, psmem, s, a));
            if (mma) RNB_TRY(launch_latent_attend_mma(s, (const bf16 *)b.qf, (const bf16 *)R.cache, d, m.scale, pos_dev, b.part, n, chunks));
            else RNB_TRY(launch_latent_attend<bf16>(s, b.qf, (const bf16 *)R.cache, d, m.scale, pos_dev, b.part, n, chunks));
        }
        // a few CTAs per head share its value rows
        const int split = n <= SMALL ? std::max(1, std::min((m.vdim + 15) / 16, 2 * sm_ / std::max(1, m.heads * n))) : 1;
        const int rows = (m.vdim + split - 1) / split;
        const dim3 og((unsigned)m.heads, (unsigned)n, (unsigned)split);
        const size_t smem = ((size_t)5 * ((m.kv_rank + 3) & ~3) + chunks) * 4;
        if (nb) RNB_CU(launch_k(latent_output_kernel<bf16>, og, dim3(LO_THREADS), smem, s, (const float *)b.part, reinterpret_cast<const bf16 *>(M.uv.w), d, chunks, pos_dev, rows, (bf16 *)act_of(b, M, n), L.out_cols, m.out_scale));
        else RNB_CU(launch_k(latent_output_kernel<float>, og, dim3(LO_THREADS), smem, s, (const float *)b.part, reinterpret_cast<const bf16 *>(M.uv.w), d, chunks, pos_dev, rows, (float *)act_of(b, M, n), L.out_cols, m.out_scale));
        return RNB_B200_OK;
    }
    RNB_CU(launch_k(latent_append_kernel<bf16>, dim3((unsigned)n), dim3(128), 0, s, (const float *)b.z, (const float *)M.dkv_norm, cfg.norm_eps, d, rot, pos_dev, (bf16 *)R.cache));
    if (rot.table) {
        RotateArgs r;
        memset(&r, 0, sizeof(r));
        r.x[0] = b.p[0];
        r.mul[0] = 1.f;
        r.heads = m.heads, r.hd = m.dim + m.rot_dim, r.off = m.dim;
        r.rot = rot;
        r.pos0 = pos_dev;
        RNB_CU(launch_k(rotate_heads_kernel<bf16>, dim3((unsigned)n, 1), dim3(256), 0, s, r));
    }
    // keys and values of every position so far, expanded from the cache rows
    const Mm ex[2] = {{&M.uk, nullptr, R.cache, (size_t)d.ld, b.kn, false}, {&M.uv, nullptr, R.cache, (size_t)d.ld, b.vx, false}};
    RNB_TRY(matmul(s, pos_host + n, ex, 2, err));
    CausalAttentionArgs a;
    memset(&a, 0, sizeof(a));
    a.q = (const bf16 *)b.p[0], a.k = (const bf16 *)b.kn, a.k2 = (const bf16 *)R.cache + m.kv_rank, a.v = (const bf16 *)b.vx;
    a.act = (bf16 *)act_of(b, M, n);
    a.pos0 = pos_dev, a.scale = m.scale, a.out_mul = m.out_scale;
    a.ldq = (size_t)m.heads * (m.dim + m.rot_dim), a.ldk = (size_t)m.heads * m.dim, a.ldk2 = (size_t)d.ld, a.ldv = (size_t)m.heads * m.vdim;
    a.tokens = n, a.heads = m.heads, a.group = 1, a.dim = m.dim, a.dim2 = m.rot_dim, a.vdim = m.vdim, a.ring = cfg.max_ctx, a.lda = L.out_cols;
    a.vec = m.dim % 8 == 0 && m.rot_dim % 8 == 0 && m.vdim % 8 == 0 && m.kv_rank % 8 == 0;
    return launch_causal_attention(s, a);
}

int LayerStack::run_mixer(cudaStream_t s, int n, StackScratch &b, StackLayer &L, int i, MixerState &R, const int *pos_dev, int pos_host, int *err) {
    switch (L.mixers[i].c.mixer) {
    case RNB_B200_MIXER_LATENT_ATTENTION: return mixer_latent(s, n, b, L, i, R, pos_dev, pos_host, err);
    case RNB_B200_MIXER_ATTENTION: return mixer_attention(s, n, b, L, i, R, pos_dev);
    case RNB_B200_MIXER_DELTA: return mixer_delta(s, n, b, L, i, R, pos_dev, err);
    default: return mixer_linear(s, n, b, L, i, R, pos_dev, err);
    }
}

int LayerStack::in_jobs(int n, StackScratch &b, StackLayer &L, Mm *jobs) {
    const size_t D = (size_t)cfg.width, stream = (size_t)n * D * (narrow(n) ? 2 : 4);
    int k = 0;
    for (size_t i = 0; i < L.mixers.size(); i++) {
        StackMixer &M = L.mixers[i];
        const char *h = (const char *)b.h;
        switch (M.c.mixer) {
        case RNB_B200_MIXER_WKV:
            jobs[k++] = {&M.r, nullptr, h, D, b.p[0], false};
            jobs[k++] = {&M.k, nullptr, h + stream, D, b.p[1], false};
            jobs[k++] = {&M.v, nullptr, h + 2 * stream, D, b.p[2], false};
            jobs[k++] = {&M.g, nullptr, h + 3 * stream, D, b.p[3], false};
            jobs[k++] = {&M.w1, nullptr, h + 4 * stream, D, b.z, true};
            break;
        case RNB_B200_MIXER_RETENTION: {
            const DenseMat *w[4] = {&M.q, &M.k, &M.v, &M.g};
            for (int j = 0; j < 4; j++) jobs[k++] = {w[j], nullptr, h, D, b.p[j], false};
            break;
        }
        case RNB_B200_MIXER_LATENT_ATTENTION:
            jobs[k++] = {&M.q, nullptr, h, D, b.p[0], absorbed(M.c, n)};
            jobs[k++] = {&M.dkv, nullptr, h, D, b.z, true};
            break;
        default:
            jobs[k++] = {&M.in, nullptr, h, D, b.p[i], false};
            if (M.c.mixer == RNB_B200_MIXER_GLA) jobs[k++] = {&M.w1, nullptr, h, D, b.aux[i], true};
            else if (M.aux_rows) jobs[k++] = {&M.aux, nullptr, h, D, b.aux[i], true};
        }
    }
    if (parallel() && L.n_ff > 0) jobs[k++] = {&L.gate, &L.up, b.h, D, (char *)b.act + (size_t)L.ff_at * (narrow(n) ? 2 : 4), false, (size_t)L.out_cols};
    return k;
}
LayerStack::Mm LayerStack::out_job(StackScratch &b, StackLayer &L) { return {&L.out, nullptr, b.act, (size_t)L.out_cols, b.y, true}; }

int LayerStack::forward(cudaStream_t s, const uint32_t *tokens_dev, int n, const int *pos_dev, int pos_host, float **x_rows, float *logits_one, float *trace, int *err) {
    StackScratch &b = scratch(n);
    if (n < 1 || n > b.cap) return fail(RNB_B200_VALIDATION_FAILED, "stack: %d tokens in one call, scratch for %d", n, b.cap);
    int cur = 0;
    RNB_CU(launch_k(dense_embed_kernel, dim3((unsigned)n), dim3(256), 0, s, reinterpret_cast<const bf16 *>(embed_.w), tokens_dev, cfg.width, cfg.embed_scale, b.x[0], b.emb));
    const float *y = nullptr, *wb = nullptr;   // the sublayer output that has not been added yet, and its norm (sandwich layers)
    const size_t D = (size_t)cfg.width;
    for (size_t i = 0; i < runs_.size(); i++) {
        LayerRun &R = runs_[i];
        StackLayer &L = layers_[R.layer];
        RNB_TRY(boundary(s, n, b, cur, y, wb, R.add_embedding, L.norm1, parallel() ? L.norm1b : nullptr, L.shifts() ? &L : nullptr, &R));
        Mm jobs[DENSE_MAX_JOBS];
        RNB_TRY(matmul(s, n, jobs, in_jobs(n, b, L, jobs), err));
        if (n <= SMALL && L.mixers.size() == 2 && L.mixers[0].c.mixer == RNB_B200_MIXER_ATTENTION && L.mixers[1].c.mixer == RNB_B200_MIXER_DELTA)
            RNB_TRY(mixers_attention_delta(s, n, b, L, R, pos_dev));
        else
            for (size_t m = 0; m < L.mixers.size(); m++) RNB_TRY(run_mixer(s, n, b, L, (int)m, R.m[m], pos_dev, pos_host, err));
        const Mm out = out_job(b, L);
        RNB_TRY(matmul(s, n, &out, 1, err));
        y = b.y, wb = parallel() ? nullptr : L.norm1b;
        if (!parallel() && L.n_ff > 0) {
            RNB_TRY(boundary(s, n, b, cur, y, wb, false, L.norm2, nullptr, nullptr, nullptr));
            const Mm gu = {&L.gate, &L.up, b.h, D, b.act, false}, down = {&L.down, nullptr, b.act, (size_t)L.n_ff, b.y, true};
            RNB_TRY(matmul(s, n, &gu, 1, err));
            RNB_TRY(matmul(s, n, &down, 1, err));
            wb = L.norm2b;
        }
        if (trace) {
            RNB_TRY(boundary(s, n, b, cur, y, wb, false, nullptr, nullptr, nullptr, nullptr));
            RNB_CU(cudaMemcpyAsync(trace + i * n * D, b.x[cur], (size_t)n * D * 4, cudaMemcpyDeviceToHost, s));
            y = wb = nullptr;
        }
    }
    if (y || logits_one) RNB_TRY(boundary(s, n, b, cur, y, wb, false, logits_one ? final_norm_ : nullptr, logits_one ? final_bias_ : nullptr, nullptr, nullptr));
    if (logits_one) {
        const Mm lm = {&embed_, nullptr, (const float *)b.h + (size_t)(n - 1) * D, D, logits_one, true};
        RNB_TRY(matmul(s, 1, &lm, 1, err));
    }
    *x_rows = b.x[cur];
    return RNB_B200_OK;
}

int LayerStack::head_rows(cudaStream_t s, const float *x, const int *rows_host, int n_rows, float *logits, int *err) {
    StackScratch &b = scratch(n_rows);
    if (n_rows < 1 || n_rows > b.cap) return fail(RNB_B200_VALIDATION_FAILED, "stack: %d logit rows, scratch for %d", n_rows, b.cap);
    RNB_CU(cudaMemcpyAsync(b.rows, rows_host, (size_t)n_rows * 4, cudaMemcpyHostToDevice, s));
    if (narrow(n_rows)) RNB_CU(launch_k(norm_rows_kernel<bf16>, dim3((unsigned)n_rows), dim3(512), 0, s, x, (const int *)b.rows, (const float *)final_norm_, (const float *)final_bias_, cfg.norm_eps, cfg.width, (bf16 *)b.h));
    else RNB_CU(launch_k(norm_rows_kernel<float>, dim3((unsigned)n_rows), dim3(512), 0, s, x, (const int *)b.rows, (const float *)final_norm_, (const float *)final_bias_, cfg.norm_eps, cfg.width, (float *)b.h));
    const Mm lm = {&embed_, nullptr, b.h, (size_t)cfg.width, logits, true};
    return matmul(s, n_rows, &lm, 1, err);
}

int LayerStack::time_matvecs(cudaStream_t s, bool count, uint64_t *bytes) {
    StackScratch &b = small_;
    const size_t D = (size_t)cfg.width;
    auto mv = [&](const Mm *j, int n) -> int {
        if (count)
            for (int i = 0; i < n; i++) *bytes += ((uint64_t)j[i].w->rows * j[i].w->cols * (j[i].w2 ? 2 : 1)) * 2 + (uint64_t)j[i].w->rows * 4 + (uint64_t)j[i].w->cols * 4;
        return matmul(s, 1, j, n, nullptr);
    };
    for (LayerRun &R : runs_) {
        StackLayer &L = layers_[R.layer];
        Mm jobs[DENSE_MAX_JOBS];
        RNB_TRY(mv(jobs, in_jobs(1, b, L, jobs)));
        const Mm o = out_job(b, L);
        RNB_TRY(mv(&o, 1));
        if (!parallel() && L.n_ff > 0) {
            const Mm gu = {&L.gate, &L.up, b.h, D, b.act, false}, down = {&L.down, nullptr, b.act, (size_t)L.n_ff, b.y, true};
            RNB_TRY(mv(&gu, 1));
            RNB_TRY(mv(&down, 1));
        }
    }
    const Mm lm = {&embed_, nullptr, b.h, D, b.logits, true};
    return mv(&lm, 1);
}

}  // namespace rnb
