// Host side of the mixed stacks: weights by name, per-run state, scratch, and the launch order of a step.
#include "layer_stack.hpp"

#include <cuda.h>
#include <math.h>

#include <algorithm>

#include "dense.cuh"
#include "latent_attention.cuh"
#include "launch.hpp"
#include "layer_glue.cuh"
#include "linear_state.cuh"

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

int LayerStack::init(const rnb_b200_mixer_cfg *layers) {
    const rnb_b200_stack_cfg &c = cfg;
    if (c.n_layer < 1 || c.width < 1 || c.vocab < 1 || c.max_ctx < 1) return fail(RNB_B200_VALIDATION_FAILED, "stack: invalid shape");
    if (c.width > 24576) return fail(RNB_B200_UNSUPPORTED, "stack: width %d exceeds 24576", c.width);
    loops_ = c.loop_times > 1;
    if (loops_ && (c.loop_start < 0 || c.loop_stop <= c.loop_start || c.loop_stop > c.n_layer)) return fail(RNB_B200_VALIDATION_FAILED, "stack: invalid loop %d .. %d", c.loop_start, c.loop_stop);
    sm_ = state().sm_count;
    layers_.resize((size_t)c.n_layer);
    for (int i = 0; i < c.n_layer; i++) {
        StackLayer &L = layers_[i];
        L.c = layers[i];
        rnb_b200_mixer_cfg &m = L.c;
        m.decay = nullptr;
        if (m.heads < 1 || m.dim < 1 || m.n_ff < 0) return fail(RNB_B200_VALIDATION_FAILED, "layer %d: invalid mixer shape", i);
        if (m.mixer == RNB_B200_MIXER_WKV) m.vdim = m.dim;
        if (m.vdim < 1) return fail(RNB_B200_VALIDATION_FAILED, "layer %d: invalid value size", i);
        const rnb_b200_rotation &r = m.rot;
        const int rotated = m.mixer == RNB_B200_MIXER_LATENT_ATTENTION ? m.rot_dim : m.dim;
        if (m.mixer != RNB_B200_MIXER_WKV && (r.dims < 0 || r.dims % 2 || r.dims > rotated || (r.dims > 0 && !(r.base > 1.0))))
            return fail(RNB_B200_VALIDATION_FAILED, "layer %d: rotation of %d dimensions does not fit %d", i, r.dims, rotated);
        if (m.mixer == RNB_B200_MIXER_WKV || m.mixer == RNB_B200_MIXER_RETENTION) {
            if (m.dim > 512) return fail(RNB_B200_UNSUPPORTED, "layer %d: state channels %d exceed 512", i, m.dim);
            if (m.mixer == RNB_B200_MIXER_RETENTION) {
                if (!layers[i].decay) return fail(RNB_B200_VALIDATION_FAILED, "layer %d: retention needs a decay per head", i);
                for (int h = 0; h < m.heads; h++) L.decay_host.push_back((float)layers[i].decay[h]);
            }
        } else if (m.mixer == RNB_B200_MIXER_LATENT_ATTENTION) {
            if (m.kv_rank < 1 || m.rot_dim < 0) return fail(RNB_B200_VALIDATION_FAILED, "layer %d: invalid latent shape", i);
            if (m.kv_rank + m.rot_dim > 1152) return fail(RNB_B200_UNSUPPORTED, "layer %d: cache row of %d exceeds 1152", i, m.kv_rank + m.rot_dim);
        } else {
            return fail(RNB_B200_UNSUPPORTED, "layer %d: unknown mixer %d", i, m.mixer);
        }
    }
    for (int i = 0; i < c.n_layer; i++) {
        StackLayer &L = layers_[i];
        if (!L.decay_host.empty()) {
            RNB_TRY(alloc((void **)&L.decay, L.decay_host.size() * 4));
            RNB_CU(cudaMemcpy(L.decay, L.decay_host.data(), L.decay_host.size() * 4, cudaMemcpyHostToDevice));
        }
        if (L.c.mixer != RNB_B200_MIXER_WKV && L.c.rot.dims > 0) RNB_TRY(rotation_table(L.c.rot, &L.rot_table));
        slots_of_layer(i);
    }
    Slot e;
    e.name = "embed", e.mat = &embed_, e.rows = c.vocab, e.cols = c.width;
    slots_.push_back(e);
    Slot f;
    f.name = "final.norm", f.vec = &final_norm_, f.rows = f.vec_total = c.width;
    slots_.push_back(f);
    const int a = loops_ ? c.loop_start : 0, b = loops_ ? c.loop_stop : 0, times = loops_ ? c.loop_times : 0;
    auto push = [&](int layer, bool emb) {
        LayerRun r;
        r.layer = layer;
        r.add_embedding = emb;
        runs_.push_back(r);
    };
    for (int i = 0; i < a; i++) push(i, false);
    for (int t = 0; t < times; t++)
        for (int i = a; i < b; i++) push(i, t > 0 && i == a);
    for (int i = b; i < c.n_layer; i++) push(i, false);
    int max_heads = 1;
    for (LayerRun &r : runs_) {
        const rnb_b200_mixer_cfg &m = layers_[r.layer].c;
        max_heads = std::max(max_heads, m.heads);
        if (m.mixer == RNB_B200_MIXER_LATENT_ATTENTION) {
            RNB_TRY(alloc(&r.cache, (size_t)c.max_ctx * latent_ld(layers_[r.layer]) * (c.f32_math ? 4 : 2)));
        } else {
            RNB_TRY(alloc((void **)&r.state, (size_t)m.heads * m.dim * m.vdim * 4));
            if (m.mixer == RNB_B200_MIXER_WKV) {
                RNB_TRY(alloc((void **)&r.shift, (size_t)c.width * 4));
                RNB_TRY(alloc((void **)&r.shift_out, (size_t)c.width * 4));
            }
        }
    }
    RNB_TRY(alloc((void **)&counters_, (size_t)max_heads * 4));
    RNB_CU(cudaMemset(counters_, 0, (size_t)max_heads * 4));
    attend_chunks_ = std::max(1, std::min((c.max_ctx + 127) / 128, 64));
    return RNB_B200_OK;
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
    if (r.scaled) {
        auto dim_of = [&](double turns) { return r.dims * log(r.original / (2.0 * M_PI * turns)) / (2.0 * log(r.base)); };
        lo = std::max(floor(dim_of(r.fast)), 0.0);
        hi = std::min(ceil(dim_of(r.slow)), (double)r.dims - 1.0);
        mult = 0.1 * log(r.factor) + 1.0;
    }
    for (int i = 0; i < half; i++) {
        f[i] = pow(r.base, -2.0 * i / r.dims);
        if (r.scaled) {
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
    const rnb_b200_mixer_cfg &m = L.c;
    const int64_t D = cfg.width, hd = (int64_t)m.heads * m.dim, hv = (int64_t)m.heads * m.vdim;
    const std::string p = "l" + std::to_string(i) + ".", x = p + "mix.";
    auto mat = [&](const std::string &name, DenseMat *dst, int64_t rows, int64_t cols) {
        Slot s;
        s.name = name, s.mat = dst, s.rows = rows, s.cols = cols;
        slots_.push_back(s);
    };
    auto vec = [&](const std::string &name, float **dst, int64_t n, float mean = 0.f, float sigma = 0.f, size_t off = 0, size_t total = 0) {
        Slot s;
        s.name = name, s.vec = dst, s.rows = n, s.vec_off = off, s.vec_total = total ? total : (size_t)n, s.synth_mean = mean, s.synth_sigma = sigma;
        slots_.push_back(s);
    };
    vec(p + "norm1", &L.norm1, D);
    vec(p + "norm1b", &L.norm1b, D);
    mat(x + "o", &L.o, D, hv);
    if (m.mixer == RNB_B200_MIXER_WKV) {
        const char *mix = "rkvgw";
        for (int j = 0; j < 5; j++) vec(x + "mu." + mix[j], &L.mu, D, 0.5f, 0.1f, (size_t)j * D, (size_t)5 * D);
        mat(x + "r", &L.r, hd, D);
        mat(x + "k", &L.k, hd, D);
        mat(x + "v", &L.v, hd, D);
        mat(x + "g", &L.g, hd, D);
        const int64_t rank = m.decay_rank > 0 ? m.decay_rank : -1;
        mat(x + "w1", &L.w1, rank, D);
        mat(x + "w2", &L.w2, hd, rank);
        vec(x + "w0", &L.w0, hd, -1.5f, 1.0f);
        vec(x + "u", &L.u, hd, 0.f, 0.5f);
        vec(x + "norm", &L.head_norm, hd, 1.f);
    } else if (m.mixer == RNB_B200_MIXER_RETENTION) {
        mat(x + "q", &L.q, hd, D);
        mat(x + "k", &L.k, hd, D);
        mat(x + "v", &L.v, hv, D);
        mat(x + "g", &L.g, hv, D);
    } else {
        mat(x + "q", &L.q, (int64_t)m.heads * (m.dim + m.rot_dim), D);
        mat(x + "dkv", &L.dkv, m.kv_rank + m.rot_dim, D);
        vec(x + "dkv.norm", &L.dkv_norm, m.kv_rank, 1.f);
        mat(x + "uk", &L.uk, hd, m.kv_rank);
        mat(x + "uv", &L.uv, hv, m.kv_rank);
    }
    if (m.n_ff > 0) {
        vec(p + "norm2", &L.norm2, D);
        vec(p + "norm2b", &L.norm2b, D);
        mat(p + "mlp.gate", &L.gate, m.n_ff, D);
        mat(p + "mlp.up", &L.up, m.n_ff, D);
        mat(p + "mlp.down", &L.down, D, m.n_ff);
    }
}

// Device storage of a tensor; rows / cols as the tensor has them.
int LayerStack::place(Slot &slot, int64_t rows, int64_t cols) {
    if (slot.vec) {
        if (!*slot.vec) {
            RNB_TRY(alloc((void **)slot.vec, slot.vec_total * 4));
            weight_bytes_ += slot.vec_total * 4;
        }
        return RNB_B200_OK;
    }
    DenseMat &m = *slot.mat;
    if (!m.w) {
        RNB_TRY(alloc((void **)&m.w, (size_t)rows * cols * 2));
        weight_bytes_ += (uint64_t)rows * cols * 2;
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
        RNB_TRY(place(*slot, slot->rows, 0));
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
        RNB_TRY(place(*slot, (int64_t)shape[0], (int64_t)shape[1]));
        RNB_CU(cudaMemcpyAsync(slot->mat->w, data, n * 2, cudaMemcpyHostToDevice, s));
        RNB_CU(cudaStreamSynchronize(s));
    }
    slot->set = true;
    return RNB_B200_OK;
}

int LayerStack::fill_synthetic(cudaStream_t s, uint64_t seed, float sigma) {
    uint64_t id = seed * 1000003ull;
    for (Slot &t : slots_) {
        const int64_t rows = t.rows < 0 ? 64 : t.rows, cols = t.cols < 0 ? 64 : t.cols;
        RNB_TRY(place(t, rows, cols));
        if (t.vec) RNB_TRY(synth_dense<float>(s, *t.vec + t.vec_off, (size_t)rows, ++id, t.synth_mean, t.synth_sigma));
        else RNB_TRY(synth_dense<bf16>(s, reinterpret_cast<bf16 *>(t.mat->w), (size_t)rows * cols, ++id, 0.f, sigma));
        t.set = true;
    }
    RNB_CU(cudaStreamSynchronize(s));
    return RNB_B200_OK;
}

int LayerStack::fill_state_synthetic(cudaStream_t s, int n_pos, uint64_t seed) {
    RNB_TRY(reset(s));
    uint64_t id = seed * 131ull;
    for (LayerRun &r : runs_) {
        const StackLayer &L = layers_[r.layer];
        if (r.cache) {
            const size_t n = (size_t)n_pos * latent_ld(L);
            if (cfg.f32_math) RNB_TRY(synth_dense<float>(s, (float *)r.cache, n, ++id, 0.f, 1.f));
            else RNB_TRY(synth_dense<bf16>(s, (bf16 *)r.cache, n, ++id, 0.f, 1.f));
        } else if (n_pos > 0) {
            RNB_TRY(synth_dense<float>(s, r.state, (size_t)L.c.heads * L.c.dim * L.c.vdim, ++id, 0.f, 1.f));
            if (r.shift) RNB_TRY(synth_dense<float>(s, r.shift, (size_t)cfg.width, ++id, 0.f, 1.f));
        }
    }
    RNB_CU(cudaStreamSynchronize(s));
    return RNB_B200_OK;
}

// ---- scratch --------------------------------------------------------------------------------------
bool LayerStack::absorbed(const StackLayer &L, int n) const {
    if (n <= SMALL || cfg.f32_math) return true;
    const rnb_b200_mixer_cfg &m = L.c;
    const LatentDims d{m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, latent_ld(L)};
    return m.vdim > 256 || latent_prefill_smem(d, la_pad16(m.vdim) <= 32 ? 32 : round_pow2(m.vdim)) > 227 * 1024;
}

int LayerStack::piece() const {
    int p = cfg.f32_math ? 512 : 4096;
    for (const StackLayer &L : layers_)
        if (L.c.mixer == RNB_B200_MIXER_LATENT_ATTENTION && absorbed(L, SMALL + 1)) p = 512;
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
// CTAs that work on one chunk of tokens
static int linear_ctas(const rnb_b200_mixer_cfg &m) { const int w = 16 * linear_tile_warps(m.vdim); return m.heads * ((m.vdim + w - 1) / w); }

int LayerStack::alloc_scratch(StackScratch &b, int cap) {
    for (void *p : b.allocs) cudaFree(p);
    b = StackScratch();
    const bool small = cap <= SMALL;
    const size_t T = (size_t)cap, D = (size_t)cfg.width, es = narrow(cap) ? 2 : 4;
    size_t proj = 1, zw = 1, ww = 1, ow = 1, aw = 1, streams = 1, qfw = 0, partw = 0, st = 0, dc = 0, kn = 0, vx = 0;
    for (const StackLayer &L : layers_) {
        const rnb_b200_mixer_cfg &m = L.c;
        const size_t hd = (size_t)m.heads * m.dim, hv = (size_t)m.heads * m.vdim;
        aw = std::max(aw, std::max(hv, (size_t)m.n_ff));
        if (m.mixer == RNB_B200_MIXER_LATENT_ATTENTION) {
            proj = std::max(proj, (size_t)m.heads * (m.dim + m.rot_dim) * (absorbed(L, cap) && es == 2 ? 2 : 1));
            zw = std::max(zw, (size_t)(m.kv_rank + m.rot_dim));
            if (absorbed(L, cap)) {
                qfw = std::max(qfw, (size_t)m.heads * (m.kv_rank + m.rot_dim + 32));
                partw = std::max(partw, (size_t)m.heads * (small ? attend_chunks_ : 1) * latent_part_ld(m.kv_rank));
            } else {
                kn = std::max(kn, (size_t)cfg.max_ctx * hd);
                vx = std::max(vx, (size_t)cfg.max_ctx * hv);
            }
        } else {
            proj = std::max(proj, std::max(hd, hv));
            ow = std::max(ow, hv);
            if (m.mixer == RNB_B200_MIXER_WKV) {
                streams = 5;
                zw = std::max(zw, (size_t)L.w1.rows);
                ww = std::max(ww, hd);
            }
            if (!small) {
                size_t nc = 1;   // most chunks any token count up to cap can have
                for (int t = 1; t <= cap; t++) {
                    const int c = linear_chunk(t, linear_ctas(m));
                    nc = std::max(nc, (size_t)((t + c - 1) / c));
                }
                st = std::max(st, nc * hd * m.vdim);
                dc = std::max(dc, nc * hd);
            }
        }
    }
    auto get = [&](void *pp, size_t bytes) -> int { return bytes ? alloc((void **)pp, bytes, &b.allocs) : RNB_B200_OK; };
    for (int i = 0; i < 2; i++) RNB_TRY(get(&b.x[i], T * D * 4));
    if (loops_) RNB_TRY(get(&b.emb, T * D * 4));
    RNB_TRY(get(&b.h, T * D * streams * es));
    for (int i = 0; i < 4; i++) RNB_TRY(get(&b.p[i], T * proj * es));
    RNB_TRY(get(&b.y, T * D * 4));
    RNB_TRY(get(&b.z, T * zw * 4));
    if (!small) RNB_TRY(get(&b.w, T * ww * 4));
    RNB_TRY(get(&b.o, T * ow * 4));
    RNB_TRY(get(&b.act, T * aw * es));
    RNB_TRY(get(&b.qf, T * qfw * 4));
    RNB_TRY(get(&b.part, T * partw * 4));
    RNB_TRY(get(&b.starts, st * 4));
    RNB_TRY(get(&b.decays, dc * 4));
    if (!small && narrow(cap) && streams == 5) RNB_TRY(get(&b.th, T * zw * 2 * 2));
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
    for (size_t i = 0; i < layers_.size(); i++) {
        const StackLayer &L = layers_[i];
        if (L.c.mixer == RNB_B200_MIXER_WKV && L.w1.rows != L.w2.cols) return fail(RNB_B200_VALIDATION_FAILED, "layer %zu: w1 has %d rows, w2 %d columns", i, L.w1.rows, L.w2.cols);
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
                         (const void *)residual_norm_kernel<bf16, 1>, (const void *)dense_gemm_kernel, (const void *)linear_state_chunk_kernel<float, false, false>,
                         (const void *)linear_state_chunk_kernel<float, false, true>, (const void *)linear_state_chunk_kernel<float, true, false>,
                         (const void *)linear_state_chunk_kernel<float, true, true>, (const void *)linear_state_chunk_kernel<bf16, false, false>,
                         (const void *)linear_state_chunk_kernel<bf16, false, true>, (const void *)linear_state_chunk_kernel<bf16, true, false>,
                         (const void *)linear_state_chunk_kernel<bf16, true, true>, (const void *)decay_rows_kernel, (const void *)linear_state_step_kernel<4>,
                         (const void *)linear_state_step_kernel<8>, (const void *)linear_state_step_kernel<16>, (const void *)linear_state_step_kernel<32>,
                         (const void *)linear_state_step_kernel<64>, (const void *)latent_prefill_kernel<4>, (const void *)latent_prefill_kernel<8>,
                         (const void *)latent_prefill_kernel<16>, (const void *)latent_prefill_kernel<32>};
    for (const void *f : fns) RNB_TRY(raise(f));
    const void *tile[] = {
#define RNB_LT(DT) (const void *)linear_state_tile_kernel<DT, false, false>, (const void *)linear_state_tile_kernel<DT, false, true>, \
                   (const void *)linear_state_tile_kernel<DT, true, false>, (const void *)linear_state_tile_kernel<DT, true, true>
        RNB_LT(2), RNB_LT(4), RNB_LT(8), RNB_LT(16)
#undef RNB_LT
    };
    for (const void *f : tile) RNB_TRY(raise(f));
    const void *lat[] = {(const void *)latent_attend_mma_kernel<1>, (const void *)latent_attend_mma_kernel<2>, (const void *)latent_attend_mma_kernel<4>,
                         (const void *)latent_attend_mma_kernel<8>, (const void *)latent_attend_mma_kernel<10>, (const void *)latent_prepare_kernel<float, float>,
                         (const void *)latent_prepare_kernel<bf16, float>, (const void *)latent_prepare_kernel<bf16, bf16>, (const void *)latent_output_kernel<float>, (const void *)latent_output_kernel<bf16>};
    for (const void *f : lat) RNB_TRY(raise(f));
    for (StackLayer &L : layers_)
        if (L.w2.w && L.w2.cols % 4 == 0 && !cfg.f32_math) {
            DenseMat &m = L.w2x;
            const size_t pitch = (size_t)L.w2.cols * 2;
            RNB_TRY(alloc((void **)&m.w, (size_t)L.w2.rows * pitch * 2));
            for (int half = 0; half < 2; half++)
                RNB_CU(cudaMemcpy2DAsync((char *)m.w + half * pitch, 2 * pitch, L.w2.w, pitch, pitch, (size_t)L.w2.rows, cudaMemcpyDeviceToDevice, s));
            m.rows = L.w2.rows;
            m.cols = 2 * L.w2.cols;
            m.tiled = true;
            PgTensorMap t;
            RNB_TRY(encode_token_map(&t, m.w, (size_t)m.rows, (size_t)m.cols, (size_t)m.cols, 64));
            memcpy(m.map, &t, sizeof(m.map));
        }
    RNB_TRY(alloc_scratch(small_, SMALL));
    RNB_TRY(reset(s));
    ready_ = true;
    return RNB_B200_OK;
}

int LayerStack::reset(cudaStream_t s) {
    for (LayerRun &r : runs_) {
        const rnb_b200_mixer_cfg &m = layers_[r.layer].c;
        if (r.state) RNB_CU(cudaMemsetAsync(r.state, 0, (size_t)m.heads * m.dim * m.vdim * 4, s));
        if (r.shift) RNB_CU(cudaMemsetAsync(r.shift, 0, (size_t)cfg.width * 4, s));
    }
    return RNB_B200_OK;
}

uint64_t LayerStack::cache_bytes_per_pos() const {
    uint64_t n = 0;
    for (const LayerRun &r : runs_)
        if (r.cache) n += (uint64_t)latent_ld(layers_[r.layer]) * (cfg.f32_math ? 4 : 2);
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
            j.cta0 = ctas;
            j.vec = jobs[i].w->cols % 8 == 0 && ((uintptr_t)j.x & 15) == 0;
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
            j.rows = j.ld = jobs[i].w->rows;
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
        j.rows = j.ld = jobs[i].w->rows;
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
int LayerStack::boundary(cudaStream_t s, int n, StackScratch &b, int &cur, const float *y, const float *wb, bool emb, const float *wn, const StackLayer *shift, LayerRun *run) {
    ResidualNormArgs a;
    memset(&a, 0, sizeof(a));
    a.x_in = a.x_out = b.x[cur];
    a.y = y;
    a.wb = wb;
    a.emb = emb ? b.emb : nullptr;
    a.wn = wn;
    a.h = b.h;
    a.mult = cfg.residual_mult;
    a.eps = cfg.norm_eps;
    a.width = cfg.width;
    a.tokens = n;
    a.rows_per_cta = shift ? 8 : 1;
    if (shift) {
        a.mu = shift->mu;
        a.n_mix = 5;
        a.shift_in = run->shift;
        a.shift_out = n <= a.rows_per_cta ? run->shift : run->shift_out;
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
    if (shift && a.shift_out != a.shift_in) RNB_CU(cudaMemcpyAsync(run->shift, run->shift_out, (size_t)cfg.width * 4, cudaMemcpyDeviceToDevice, s));
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
template <int DT>
static int launch_linear_tiles(cudaStream_t s, const LinearChunkArgs &a) {
    const int nw = linear_tile_warps(a.vdim);
    const unsigned zb = (unsigned)((a.vdim + 16 * nw - 1) / (16 * nw));
    const size_t smem = linear_tile_smem(DT, nw).bytes;
    const dim3 block((unsigned)(32 * nw));
    if (a.n_chunks > 1) {
        const dim3 grid((unsigned)(a.n_chunks - 1), (unsigned)a.heads, zb);
        if (a.w) RNB_CU(launch_k(linear_state_tile_kernel<DT, false, false>, grid, block, smem, s, a));
        else RNB_CU(launch_k(linear_state_tile_kernel<DT, false, true>, grid, block, smem, s, a));
        RNB_TRY(launch_linear_scan(s, a));
    }
    const dim3 grid((unsigned)a.n_chunks, (unsigned)a.heads, zb);
    if (a.w) RNB_CU(launch_k(linear_state_tile_kernel<DT, true, false>, grid, block, smem, s, a));
    else RNB_CU(launch_k(linear_state_tile_kernel<DT, true, true>, grid, block, smem, s, a));
    return RNB_B200_OK;
}
template <class AT>
static int launch_linear_chunks(cudaStream_t s, LinearChunkArgs a) {
    const bool cw = a.w == nullptr;
    a.G = round_pow2((a.dim + LS_TI - 1) / LS_TI);
    a.JG = std::min((a.vdim + 3) / 4, 256 / a.G);
    const dim3 block((unsigned)((a.G * a.JG + 31) / 32 * 32));
    const unsigned zb = (unsigned)((a.vdim + 4 * a.JG - 1) / (4 * a.JG));
    const size_t smem = linear_chunk_smem(a.G, a.JG);
    if (a.n_chunks > 1) {
        const dim3 grid((unsigned)(a.n_chunks - 1), (unsigned)a.heads, zb);
        if (cw) RNB_CU(launch_k(linear_state_chunk_kernel<AT, false, true>, grid, block, smem, s, a));
        else RNB_CU(launch_k(linear_state_chunk_kernel<AT, false, false>, grid, block, smem, s, a));
        RNB_TRY(launch_linear_scan(s, a));
    }
    const dim3 grid((unsigned)a.n_chunks, (unsigned)a.heads, zb);
    if (cw) RNB_CU(launch_k(linear_state_chunk_kernel<AT, true, true>, grid, block, smem, s, a));
    else RNB_CU(launch_k(linear_state_chunk_kernel<AT, true, false>, grid, block, smem, s, a));
    return RNB_B200_OK;
}
template <class HT>
static int launch_head_norm_gate(cudaStream_t s, const float *o, const float *w, const void *g, float eps, int n, int heads, int vdim, void *act) {
    const int v = vdim % 4 == 0 ? 4 : 1, lanes = std::min(32, round_pow2((vdim + v - 1) / v));
    const size_t units = (size_t)n * heads;
    const dim3 grid((unsigned)((units * lanes + 255) / 256));
    if (v == 4) RNB_CU(launch_k(head_norm_gate_kernel<HT, HT, 4>, grid, dim3(256), 0, s, o, w, (const HT *)g, eps, units, heads, vdim, lanes, (HT *)act));
    else RNB_CU(launch_k(head_norm_gate_kernel<HT, HT, 1>, grid, dim3(256), 0, s, o, w, (const HT *)g, eps, units, heads, vdim, lanes, (HT *)act));
    return RNB_B200_OK;
}

// Time mixing and retention: projections, recurrence, head norm and gate; the result is the input of W_o in b.act.
int LayerStack::mixer_linear(cudaStream_t s, int n, StackScratch &b, StackLayer &L, LayerRun &R, const int *pos_dev, int *err) {
    const rnb_b200_mixer_cfg &m = L.c;
    const bool wkv = m.mixer == RNB_B200_MIXER_WKV, nb = narrow(n);
    const size_t D = (size_t)cfg.width, stream = (size_t)n * D * (nb ? 2 : 4);
    const char *h = (const char *)b.h;
    auto in = [&](int i) -> const void * { return wkv ? h + i * stream : h; };
    const Mm jobs[5] = {{wkv ? &L.r : &L.q, nullptr, in(0), D, b.p[0], false}, {&L.k, nullptr, in(1), D, b.p[1], false}, {&L.v, nullptr, in(2), D, b.p[2], false},
                        {&L.g, nullptr, in(3), D, b.p[3], false}, {&L.w1, nullptr, in(4), D, b.z, true}};
    RNB_TRY(matmul(s, n, jobs, wkv ? 5 : 4, err));
    const Rotation rot{(const float2 *)L.rot_table, m.rot.dims, m.rot.interleaved};
    const float k_mul = wkv ? 1.f : 1.f / sqrtf((float)m.dim);
    if (n <= SMALL) {
        LinearStepArgs a;
        memset(&a, 0, sizeof(a));
        a.r = (const float *)b.p[0], a.k = (const float *)b.p[1], a.v = (const float *)b.p[2], a.g = (const float *)b.p[3];
        a.z = b.z, a.w0 = L.w0, a.decay = L.decay, a.u = L.u;
        a.w2 = reinterpret_cast<const bf16 *>(L.w2.w);
        a.norm = L.head_norm;
        a.rot = rot;
        a.pos0 = pos_dev;
        a.k_mul = k_mul, a.eps = cfg.norm_eps;
        a.state = R.state, a.o = b.o, a.act = (float *)b.act;
        a.counters = counters_;
        a.tokens = n, a.heads = m.heads, a.dim = m.dim, a.vdim = m.vdim, a.rank = wkv ? L.w1.rows : 0;
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
    if (wkv) {
        const int ch = m.heads * m.dim, rank = L.w1.rows;
        if (nb && L.w2x.w) {
            const size_t nz = (size_t)n * rank;
            RNB_CU(launch_k(tanh_split_kernel, dim3((unsigned)((nz + 255) / 256)), dim3(256), 0, s, (const float *)b.z, rank, nz, reinterpret_cast<bf16 *>(b.th)));
            const Mm dj = {&L.w2x, nullptr, b.th, (size_t)2 * rank, b.w, true, L.w0};
            RNB_TRY(matmul(s, n, &dj, 1, err));
        } else
            RNB_CU(launch_k(decay_rows_kernel, dim3((unsigned)((ch + 127) / 128), (unsigned)((n + 15) / 16)), dim3(128), (size_t)rank * 64, s, (const float *)b.z,
                        reinterpret_cast<const bf16 *>(L.w2.w), (const float *)L.w0, n, rank, ch, b.w));
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
    a.r = b.p[0], a.k = b.p[1], a.v = b.p[2];
    a.w = wkv ? b.w : nullptr;
    a.decay = L.decay, a.u = L.u;
    a.state = R.state, a.o = b.o, a.starts = b.starts, a.decays = b.decays;
    a.tokens = n, a.heads = m.heads, a.dim = m.dim, a.vdim = m.vdim;
    a.chunk = linear_chunk(n, linear_ctas(m));
    a.n_chunks = (n + a.chunk - 1) / a.chunk;
    if (nb) {
        if (!linear_tiled(m)) RNB_TRY(launch_linear_chunks<bf16>(s, a));
        else if (m.dim <= 32) RNB_TRY(launch_linear_tiles<2>(s, a));
        else if (m.dim <= 64) RNB_TRY(launch_linear_tiles<4>(s, a));
        else if (m.dim <= 128) RNB_TRY(launch_linear_tiles<8>(s, a));
        else RNB_TRY(launch_linear_tiles<16>(s, a));
        return launch_head_norm_gate<bf16>(s, b.o, L.head_norm, b.p[3], cfg.norm_eps, n, m.heads, m.vdim, b.act);
    }
    RNB_TRY(launch_linear_chunks<float>(s, a));
    return launch_head_norm_gate<float>(s, b.o, L.head_norm, b.p[3], cfg.norm_eps, n, m.heads, m.vdim, b.act);
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

int LayerStack::mixer_latent(cudaStream_t s, int n, StackScratch &b, StackLayer &L, LayerRun &R, const int *pos_dev, int pos_host, int *err) {
    const rnb_b200_mixer_cfg &m = L.c;
    const size_t D = (size_t)cfg.width;
    const LatentDims d{m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, latent_ld(L)};
    const Rotation rot{(const float2 *)L.rot_table, m.rot.dims, m.rot.interleaved};
    const bool ab = absorbed(L, n), nb = narrow(n);
    const Mm jobs[2] = {{&L.q, nullptr, b.h, D, b.p[0], ab}, {&L.dkv, nullptr, b.h, D, b.z, true}};
    RNB_TRY(matmul(s, n, jobs, 2, err));
    if (ab) {
        LatentPrepareArgs a;
        memset(&a, 0, sizeof(a));
        a.q = (const float *)b.p[0], a.y = b.z, a.w = L.dkv_norm;
        a.uk = reinterpret_cast<const bf16 *>(L.uk.w);
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
        if (nb) RNB_CU(launch_k(latent_output_kernel<bf16>, og, dim3(LO_THREADS), smem, s, (const float *)b.part, reinterpret_cast<const bf16 *>(L.uv.w), d, chunks, pos_dev, rows, (bf16 *)b.act));
        else RNB_CU(launch_k(latent_output_kernel<float>, og, dim3(LO_THREADS), smem, s, (const float *)b.part, reinterpret_cast<const bf16 *>(L.uv.w), d, chunks, pos_dev, rows, (float *)b.act));
        return RNB_B200_OK;
    }
    RNB_CU(launch_k(latent_append_kernel<bf16>, dim3((unsigned)n), dim3(128), 0, s, (const float *)b.z, (const float *)L.dkv_norm, cfg.norm_eps, d, rot, pos_dev, (bf16 *)R.cache));
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
    const Mm ex[2] = {{&L.uk, nullptr, R.cache, (size_t)d.ld, b.kn, false}, {&L.uv, nullptr, R.cache, (size_t)d.ld, b.vx, false}};
    RNB_TRY(matmul(s, pos_host + n, ex, 2, err));
    LatentPrefillArgs a;
    memset(&a, 0, sizeof(a));
    a.q = (const bf16 *)b.p[0], a.kn = (const bf16 *)b.kn, a.kr = (const bf16 *)R.cache + m.kv_rank, a.v = (const bf16 *)b.vx;
    a.act = (bf16 *)b.act;
    a.pos0 = pos_dev, a.scale = m.scale, a.tokens = n, a.d = d;
    a.vec = m.dim % 8 == 0 && m.rot_dim % 8 == 0 && m.vdim % 8 == 0 && m.kv_rank % 8 == 0;
    const dim3 grid((unsigned)((n + LA_ROWS - 1) / LA_ROWS), (unsigned)m.heads), block(LA_THREADS);
    if (m.vdim <= 32) RNB_CU(launch_k(latent_prefill_kernel<4>, grid, block, latent_prefill_smem(d, 32), s, a));
    else if (m.vdim <= 64) RNB_CU(launch_k(latent_prefill_kernel<8>, grid, block, latent_prefill_smem(d, 64), s, a));
    else if (m.vdim <= 128) RNB_CU(launch_k(latent_prefill_kernel<16>, grid, block, latent_prefill_smem(d, 128), s, a));
    else RNB_CU(launch_k(latent_prefill_kernel<32>, grid, block, latent_prefill_smem(d, 256), s, a));
    return RNB_B200_OK;
}

int LayerStack::forward(cudaStream_t s, const uint32_t *tokens_dev, int n, const int *pos_dev, int pos_host, float **x_rows, float *logits_one, float *trace, int *err) {
    StackScratch &b = scratch(n);
    if (n < 1 || n > b.cap) return fail(RNB_B200_VALIDATION_FAILED, "stack: %d tokens in one call, scratch for %d", n, b.cap);
    int cur = 0;
    RNB_CU(launch_k(dense_embed_kernel, dim3((unsigned)n), dim3(256), 0, s, reinterpret_cast<const bf16 *>(embed_.w), tokens_dev, cfg.width, b.x[0], b.emb));
    const float *y = nullptr, *wb = nullptr;   // the sublayer output that has not been added yet, and its norm
    const size_t D = (size_t)cfg.width;
    for (size_t i = 0; i < runs_.size(); i++) {
        LayerRun &R = runs_[i];
        StackLayer &L = layers_[R.layer];
        const bool shift = L.c.mixer == RNB_B200_MIXER_WKV;
        RNB_TRY(boundary(s, n, b, cur, y, wb, R.add_embedding, L.norm1, shift ? &L : nullptr, &R));
        if (L.c.mixer == RNB_B200_MIXER_LATENT_ATTENTION) RNB_TRY(mixer_latent(s, n, b, L, R, pos_dev, pos_host, err));
        else RNB_TRY(mixer_linear(s, n, b, L, R, pos_dev, err));
        const Mm out = {&L.o, nullptr, b.act, (size_t)L.o.cols, b.y, true};
        RNB_TRY(matmul(s, n, &out, 1, err));
        y = b.y, wb = L.norm1b;
        if (L.c.n_ff > 0) {
            RNB_TRY(boundary(s, n, b, cur, y, wb, false, L.norm2, nullptr, nullptr));
            const Mm gu = {&L.gate, &L.up, b.h, D, b.act, false}, down = {&L.down, nullptr, b.act, (size_t)L.c.n_ff, b.y, true};
            RNB_TRY(matmul(s, n, &gu, 1, err));
            RNB_TRY(matmul(s, n, &down, 1, err));
            wb = L.norm2b;
        }
        if (trace) {
            RNB_TRY(boundary(s, n, b, cur, y, wb, false, nullptr, nullptr, nullptr));
            RNB_CU(cudaMemcpyAsync(trace + i * n * D, b.x[cur], (size_t)n * D * 4, cudaMemcpyDeviceToHost, s));
            y = wb = nullptr;
        }
    }
    if (y || logits_one) RNB_TRY(boundary(s, n, b, cur, y, wb, false, logits_one ? final_norm_ : nullptr, nullptr, nullptr));
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
    if (narrow(n_rows)) RNB_CU(launch_k(norm_rows_kernel<bf16>, dim3((unsigned)n_rows), dim3(512), 0, s, x, (const int *)b.rows, (const float *)final_norm_, cfg.norm_eps, cfg.width, (bf16 *)b.h));
    else RNB_CU(launch_k(norm_rows_kernel<float>, dim3((unsigned)n_rows), dim3(512), 0, s, x, (const int *)b.rows, (const float *)final_norm_, cfg.norm_eps, cfg.width, (float *)b.h));
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
        if (L.c.mixer == RNB_B200_MIXER_LATENT_ATTENTION) {
            const Mm j[2] = {{&L.q, nullptr, b.h, D, b.p[0], true}, {&L.dkv, nullptr, b.h, D, b.z, true}};
            RNB_TRY(mv(j, 2));
        } else {
            const bool wkv = L.c.mixer == RNB_B200_MIXER_WKV;
            const Mm j[5] = {{wkv ? &L.r : &L.q, nullptr, b.h, D, b.p[0], true}, {&L.k, nullptr, b.h, D, b.p[1], true}, {&L.v, nullptr, b.h, D, b.p[2], true},
                             {&L.g, nullptr, b.h, D, b.p[3], true}, {&L.w1, nullptr, b.h, D, b.z, true}};
            RNB_TRY(mv(j, wkv ? 5 : 4));
        }
        const Mm o = {&L.o, nullptr, b.act, (size_t)L.o.cols, b.y, true};
        RNB_TRY(mv(&o, 1));
        if (L.c.n_ff > 0) {
            const Mm gu = {&L.gate, &L.up, b.h, D, b.act, false}, down = {&L.down, nullptr, b.act, (size_t)L.c.n_ff, b.y, true};
            RNB_TRY(mv(&gu, 1));
            RNB_TRY(mv(&down, 1));
        }
    }
    const Mm lm = {&embed_, nullptr, b.h, D, b.logits, true};
    return mv(&lm, 1);
}

}  // namespace rnb
