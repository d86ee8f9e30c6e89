// Softmax attention with grouped key/value heads, an optional window, rotated (and optionally
// root-mean-square normed) queries and keys, and an optional sigmoid gate per head.  Keys and values live in
// rings: position p in row p % ring of [ring][kv_heads * dim] and [ring][kv_heads * vdim].
//
//   attention_prepare_kernel   many tokens: rotation and norm of queries and keys, append to the rings
//   causal_attention_kernel    then runs over the rings (bf16, tensor cores; causal_attention.cuh)
//   attention_step_kernel      1..8 tokens, one launch: rotation, norm, append, attention split over the
//                              visible keys, merge, gate.  With fresh = 0 it reads prepared rings only (prompts in f32).
#pragma once
#include "causal_attention.cuh"
#include "linear_state.cuh"

namespace rnb {

struct WindowAttentionArgs {
    const void *q, *k, *v;     // projections (AT): token t's rows at + t * ld
    void *qn;                  // prepare: the finished queries (AT) [tokens][heads * dim]
    void *kc, *vc;             // rings (CT)
    const float *gate;         // null or [tokens][ldg], one value per head
    float *part;               // step: [tokens][kv_heads][chunks][rep * (vdim + 2)]
    int *counters;             // step: [tokens][kv_heads], zero between launches
    void *act;                 // step: output (AT), rows of lda
    const int *pos0;
    Rotation rot;
    float eps, scale, out_mul;
    int tokens, heads, kv_heads, dim, vdim, ld, ldg, lda, ring, window, qk_norm, fresh;
};

// One warp: store(e, value) for every element of the rotated (and normed) vector x.
template <class AT, class Store>
__device__ __forceinline__ void rotated_normed_row(const AT *x, const Rotation &rot, int pos, int dim, bool norm, float eps, Store store) {
    const int lane = threadIdx.x & 31;
    auto at = [&](int e) { return rotated_element(rot, pos, e, [&](int i) { return to_f32(x[i]); }); };
    if (dim <= 256) {
        float v[8], ss = 0.f;
#pragma unroll
        for (int i = 0; i < 8; i++) {
            const int e = lane + 32 * i;
            v[i] = e < dim ? at(e) : 0.f;
            ss = fmaf(v[i], v[i], ss);
        }
        const float r = norm ? 1.0f / sqrtf(warp_sum(ss) / (float)dim + eps) : 1.0f;
#pragma unroll
        for (int i = 0; i < 8; i++)
            if (lane + 32 * i < dim) store(lane + 32 * i, v[i] * r);
    } else {
        float ss = 0.f;
        for (int e = lane; e < dim; e += 32) {
            const float v = at(e);
            ss = fmaf(v, v, ss);
        }
        const float r = norm ? 1.0f / sqrtf(warp_sum(ss) / (float)dim + eps) : 1.0f;
        for (int e = lane; e < dim; e += 32) store(e, at(e) * r);
    }
}

// grid = (tokens, ceil((heads + 2 kv_heads) / 8)), 256 threads: a warp per query, key or value vector
template <class AT, class CT>
RNB_GLOBAL void __launch_bounds__(256)
attention_prepare_kernel(const __grid_constant__ WindowAttentionArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, unit = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, pos = *a.pos0 + t;
    if (unit >= a.heads + 2 * a.kv_heads) return;
    const size_t row = (size_t)t * a.ld, slot = (size_t)(pos % a.ring);
    if (unit < a.heads) {
        AT *out = reinterpret_cast<AT *>(a.qn) + ((size_t)t * a.heads + unit) * a.dim;
        rotated_normed_row(reinterpret_cast<const AT *>(a.q) + row + (size_t)unit * a.dim, a.rot, pos, a.dim, a.qk_norm, a.eps, [&](int e, float v) { out[e] = from_f32<AT>(v); });
    } else if (unit < a.heads + a.kv_heads) {
        const int g = unit - a.heads;
        CT *out = reinterpret_cast<CT *>(a.kc) + (slot * a.kv_heads + g) * a.dim;
        rotated_normed_row(reinterpret_cast<const AT *>(a.k) + row + (size_t)g * a.dim, a.rot, pos, a.dim, a.qk_norm, a.eps, [&](int e, float v) { out[e] = from_f32<CT>(v); });
    } else {
        const int g = unit - a.heads - a.kv_heads;
        const AT *src = reinterpret_cast<const AT *>(a.v) + row + (size_t)g * a.vdim;
        CT *out = reinterpret_cast<CT *>(a.vc) + (slot * a.kv_heads + g) * a.vdim;
        for (int e = lane; e < a.vdim; e += 32) out[e] = from_f32<CT>(to_f32(src[e]));
    }
}

// A step CTA: 64 keys at a time of one key/value head, for the rep query heads that share it.
constexpr int AS_KEYS = 64, AS_THREADS = 256;
template <class CT>
struct AttentionStepSmem {
    int kp, vp;                                // elements per staged key / value row
    uint32_t k, v, q, s, acc, stat, bytes;
};
template <class CT>
__host__ __device__ inline AttentionStepSmem<CT> attention_step_smem(int rep, int dim, int vdim) {
    constexpr int E = 16 / (int)sizeof(CT);
    AttentionStepSmem<CT> L;
    L.kp = (dim + E - 1) / E * E + E;
    L.vp = (vdim + E - 1) / E * E + E;
    L.k = 0;
    L.v = L.k + (uint32_t)(AS_KEYS * L.kp * sizeof(CT));
    L.q = L.v + (uint32_t)(AS_KEYS * L.vp * sizeof(CT));
    L.s = L.q + (uint32_t)(((size_t)rep * dim * 4 + 15) & ~(size_t)15);
    L.acc = L.s + (uint32_t)(rep * AS_KEYS * 4);
    L.stat = L.acc + (uint32_t)(((size_t)rep * vdim * 4 + 15) & ~(size_t)15);
    L.bytes = L.stat + (uint32_t)(3 * rep * 4);
    return L;
}
// keys per chunk when n of them are split over at most `chunks` CTAs
__device__ __forceinline__ int attention_chunk_keys(int n, int chunks) { return max(AS_KEYS, ((n + chunks - 1) / chunks + AS_KEYS - 1) / AS_KEYS * AS_KEYS); }

// grid = (chunks, kv_heads, tokens)
template <class AT, class CT>
RNB_GLOBAL void __launch_bounds__(AS_THREADS)
attention_step_kernel(const __grid_constant__ WindowAttentionArgs a) {
    extern __shared__ __align__(16) uint8_t as_smem[];
    pdl_launch_dependents();
    const int rep = a.heads / a.kv_heads, dim = a.dim, vdim = a.vdim, g = blockIdx.y, t = blockIdx.z, chunks = gridDim.x;
    const AttentionStepSmem<CT> L = attention_step_smem<CT>(rep, dim, vdim);
    CT *sk = reinterpret_cast<CT *>(as_smem + L.k), *sv = reinterpret_cast<CT *>(as_smem + L.v);
    float *sq = reinterpret_cast<float *>(as_smem + L.q), *ss = reinterpret_cast<float *>(as_smem + L.s), *acc = reinterpret_cast<float *>(as_smem + L.acc);
    float *s_m = reinterpret_cast<float *>(as_smem + L.stat), *s_l = s_m + rep, *s_c = s_l + rep;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    constexpr int E = 16 / (int)sizeof(CT);
    const bool vec = dim % E == 0 && vdim % E == 0;
    pdl_wait();
    const int pos0 = *a.pos0, pos = pos0 + t;
    const int n = a.window > 0 ? min(pos + 1, a.window) : pos + 1, per = attention_chunk_keys(n, chunks), active = (n + per - 1) / per;
    if ((int)blockIdx.x >= active) return;
    const int lo = pos + 1 - n + (int)blockIdx.x * per, hi = min(lo + per, pos + 1);
    const int fresh = a.fresh ? pos0 : pos + 1;   // keys from here on come from the projections
    const CT *kc = reinterpret_cast<const CT *>(a.kc) + (size_t)g * dim, *vc = reinterpret_cast<const CT *>(a.vc) + (size_t)g * vdim;
    const size_t ldk = (size_t)a.kv_heads * dim, ldv = (size_t)a.kv_heads * vdim;
    auto load = [&](int base) {
        const int cached = min(min(hi, fresh) - base, AS_KEYS);   // rows that the rings hold
        if (vec) {
            const int qk = dim / E, all = qk + vdim / E;
            for (int i = tid; i < AS_KEYS * all; i += AS_THREADS) {
                const int r = i / all, c = i % all, key = base + r;
                const bool val = c >= qk, in = r < cached;
                if (!in && key >= fresh && key < hi) continue;   // written below
                const size_t slot = (size_t)((in ? key : lo) % a.ring);
                const CT *src = val ? vc + slot * ldv + (c - qk) * E : kc + slot * ldk + c * E;
                const uint32_t dst = val ? smem_u32(sv + r * L.vp + (c - qk) * E) : smem_u32(sk + r * L.kp + c * E);
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(in ? 16u : 0u) : "memory");
            }
        } else {
            const int all = dim + vdim;
            for (int i = tid; i < AS_KEYS * all; i += AS_THREADS) {
                const int r = i / all, c = i % all, key = base + r;
                const bool in = r < cached;
                if (!in && key >= fresh && key < hi) continue;
                const size_t slot = (size_t)((in ? key : lo) % a.ring);
                if (c < dim) sk[r * L.kp + c] = in ? kc[slot * ldk + c] : from_f32<CT>(0.f);
                else sv[r * L.vp + c - dim] = in ? vc[slot * ldv + c - dim] : from_f32<CT>(0.f);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        for (int key = max(base, fresh) + warp; key < min(hi, base + AS_KEYS); key += AS_THREADS / 32) {
            const int r = key - base;
            const bool append = key == pos;   // one CTA per key/value head and token
            const size_t row = (size_t)(key - pos0) * a.ld, slot = (size_t)(key % a.ring);
            CT *ko = reinterpret_cast<CT *>(a.kc) + slot * ldk + (size_t)g * dim, *vo = reinterpret_cast<CT *>(a.vc) + slot * ldv + (size_t)g * vdim;
            rotated_normed_row(reinterpret_cast<const AT *>(a.k) + row + (size_t)g * dim, a.rot, key, dim, a.qk_norm, a.eps, [&](int e, float v) {
                const CT x = from_f32<CT>(v);
                sk[r * L.kp + e] = x;
                if (append) ko[e] = x;
            });
            const AT *src = reinterpret_cast<const AT *>(a.v) + row + (size_t)g * vdim;
            for (int e = lane; e < vdim; e += 32) {
                const CT x = from_f32<CT>(to_f32(src[e]));
                sv[r * L.vp + e] = x;
                if (append) vo[e] = x;
            }
        }
    };
    load(lo);
    for (int j = warp; j < rep; j += AS_THREADS / 32) {
        const int h = g * rep + j;
        rotated_normed_row(reinterpret_cast<const AT *>(a.q) + (size_t)t * a.ld + (size_t)h * dim, a.rot, pos, dim, a.qk_norm, a.eps, [&](int e, float v) { sq[j * dim + e] = v; });
        if (lane == 0) s_m[j] = -INFINITY, s_l[j] = 0.f;
    }
    for (int i = tid; i < rep * vdim; i += AS_THREADS) acc[i] = 0.f;
    for (int base = lo; base < hi; base += AS_KEYS) {
        const int nk = min(AS_KEYS, hi - base);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        for (int i = tid; i < rep * AS_KEYS; i += AS_THREADS) {
            const int r = i % AS_KEYS, j = i / AS_KEYS;
            float s = 0.f;
            const float *q = sq + j * dim;
            const CT *k = sk + r * L.kp;
            if (vec) {
                float s2 = 0.f;
                for (int e = 0; e < dim; e += E) {
                    const uint4 w = *reinterpret_cast<const uint4 *>(k + e);
                    const float4 x = *reinterpret_cast<const float4 *>(q + e);
                    if (E == 8) {
                        const float4 y = *reinterpret_cast<const float4 *>(q + e + 4);
                        s = fmaf(bf16_lo(w.x), x.x, s), s2 = fmaf(bf16_hi(w.x), x.y, s2);
                        s = fmaf(bf16_lo(w.y), x.z, s), s2 = fmaf(bf16_hi(w.y), x.w, s2);
                        s = fmaf(bf16_lo(w.z), y.x, s), s2 = fmaf(bf16_hi(w.z), y.y, s2);
                        s = fmaf(bf16_lo(w.w), y.z, s), s2 = fmaf(bf16_hi(w.w), y.w, s2);
                    } else {
                        s = fmaf(__uint_as_float(w.x), x.x, s), s2 = fmaf(__uint_as_float(w.y), x.y, s2);
                        s = fmaf(__uint_as_float(w.z), x.z, s), s2 = fmaf(__uint_as_float(w.w), x.w, s2);
                    }
                }
                s += s2;
            } else {
                for (int e = 0; e < dim; e++) s = fmaf(to_f32(k[e]), q[e], s);
            }
            ss[i] = r < nk ? s * a.scale : -INFINITY;
        }
        __syncthreads();
        for (int j = warp; j < rep; j += AS_THREADS / 32) {
            const float x0 = ss[j * AS_KEYS + lane], x1 = ss[j * AS_KEYS + lane + 32], old = s_m[j];
            const float m = fmaxf(old, warp_max(fmaxf(x0, x1)));
            const float p0 = expf(x0 - m), p1 = expf(x1 - m), sum = warp_sum(p0 + p1);
            ss[j * AS_KEYS + lane] = p0;
            ss[j * AS_KEYS + lane + 32] = p1;
            if (lane == 0) {
                const float c = expf(old - m);
                s_c[j] = c;
                s_m[j] = m;
                s_l[j] = fmaf(s_l[j], c, sum);
            }
        }
        __syncthreads();
        const int n4 = (nk + 3) / 4;
        if (vdim % 2 == 0) {
            for (int i = tid; i < rep * vdim / 2; i += AS_THREADS) {
                const int j = i / (vdim / 2), c = i % (vdim / 2) * 2;
                const float4 *p = reinterpret_cast<const float4 *>(ss + j * AS_KEYS);
                const CT *v = sv + c;
                float o0 = 0.f, o1 = 0.f;
                auto two = [&](int r, float w) {
                    o0 = fmaf(w, to_f32(v[r * L.vp]), o0);
                    o1 = fmaf(w, to_f32(v[r * L.vp + 1]), o1);
                };
#pragma unroll 4
                for (int r = 0; r < n4; r++) {
                    const float4 w = p[r];
                    two(4 * r, w.x), two(4 * r + 1, w.y), two(4 * r + 2, w.z), two(4 * r + 3, w.w);
                }
                acc[j * vdim + c] = fmaf(acc[j * vdim + c], s_c[j], o0);
                acc[j * vdim + c + 1] = fmaf(acc[j * vdim + c + 1], s_c[j], o1);
            }
        } else {
            for (int i = tid; i < rep * vdim; i += AS_THREADS) {
                const int j = i / vdim, c = i % vdim;
                float o = 0.f;
                for (int r = 0; r < nk; r++) o = fmaf(ss[j * AS_KEYS + r], to_f32(sv[r * L.vp + c]), o);
                acc[i] = fmaf(acc[i], s_c[j], o);
            }
        }
        __syncthreads();
        if (base + AS_KEYS < hi) load(base + AS_KEYS);
    }
    AT *act = reinterpret_cast<AT *>(a.act) + (size_t)t * a.lda;
    auto gate_of = [&](int h) { return a.gate ? a.out_mul / (1.0f + expf(-a.gate[(size_t)t * a.ldg + h])) : a.out_mul; };
    if (active == 1) {
        for (int i = tid; i < rep * vdim; i += AS_THREADS) {
            const int j = i / vdim, h = g * rep + j;
            act[(size_t)h * vdim + i % vdim] = from_f32<AT>(acc[i] / s_l[j] * gate_of(h));
        }
        return;
    }
    const size_t pl = (size_t)rep * (vdim + 2);
    float *part = a.part + ((size_t)t * a.kv_heads + g) * chunks * pl, *mine = part + blockIdx.x * pl;
    for (int i = tid; i < rep * vdim; i += AS_THREADS) __stcg(mine + i, acc[i]);
    for (int j = tid; j < rep; j += AS_THREADS) __stcg(mine + rep * vdim + j, s_m[j]), __stcg(mine + rep * (vdim + 1) + j, s_l[j]);
    if (!last_of_head(a.counters + t * a.kv_heads + g, active)) return;
    // the chunks' weights, then their weighted sum; ss is free and holds up to AS_KEYS of them per query head
    for (int j = warp; j < rep; j += AS_THREADS / 32) {
        float m = -INFINITY, l = 0.f;
        for (int c = lane; c < active; c += 32) m = fmaxf(m, __ldcg(part + c * pl + rep * vdim + j));
        m = warp_max(m);
        for (int c = lane; c < active; c += 32) {
            const float w = expf(__ldcg(part + c * pl + rep * vdim + j) - m);
            ss[j * AS_KEYS + c] = w;
            l = fmaf(w, __ldcg(part + c * pl + rep * (vdim + 1) + j), l);
        }
        l = warp_sum(l);
        if (lane == 0) s_l[j] = gate_of(g * rep + j) / l;
    }
    __syncthreads();
    for (int i = tid; i < rep * vdim; i += AS_THREADS) {
        const int j = i / vdim;
        float o = 0.f;
#pragma unroll 8
        for (int c = 0; c < active; c++) o = fmaf(ss[j * AS_KEYS + c], __ldcg(part + c * pl + i), o);
        act[(size_t)(g * rep + j) * vdim + i % vdim] = from_f32<AT>(o * s_l[j]);
    }
}

}  // namespace rnb
