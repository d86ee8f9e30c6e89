// Softmax attention with grouped key/value heads, an optional window, rotated (and optionally
// root-mean-square normed) queries and keys, and an optional sigmoid gate per head.  Keys and values live in
// rings: position p in row p % ring of [ring][kv_heads * dim] and [ring][kv_heads * vdim].
//
//   attention_prepare_kernel   many tokens: rotation and norm of queries and keys, append to the rings
//   causal_attention_kernel    then runs over the rings (bf16, tensor cores; causal_attention.cuh)
//   attention_step_kernel      1..8 tokens, one launch: rotation, norm, append, attention split over the
//                              visible keys, merge, gate.  With fresh = 0 it reads prepared rings only (prompts in f32).
//   attention_delta_step_kernel  the same and the delta rule's step (delta_rule.cuh) side by side
#pragma once
#include <type_traits>

#include "causal_attention.cuh"
#include "delta_rule.cuh"

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
    int tokens, heads, kv_heads, dim, vdim, ld, ldg, lda, ring, window, qk_norm, fresh, fours;   // fours: rotated_normed_fours applies
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

// The same for vectors whose rotated pairs (2i, 2i + 1) and accesses of four elements do not straddle anything (dim and
// rotated dims multiples of 4, rows aligned): put(e, four values) for every fourth element.
template <class AT>
struct alignas(4 * sizeof(AT)) Four { AT v[4]; };
template <class CT>
__device__ __forceinline__ void store_four(CT *p, const float (&v)[4]) {
    Four<CT> o;
#pragma unroll
    for (int q = 0; q < 4; q++) o.v[q] = from_f32<CT>(v[q]);
    *reinterpret_cast<Four<CT> *>(p) = o;
}
template <class AT, class Put>
__device__ __forceinline__ void rotated_normed_fours(const AT *x, const Rotation &rot, int pos, int dim, bool norm, float eps, Put put) {
    const float2 *table = rot.table + (size_t)pos * (rot.dims / 2);
    auto four = [&](int e, float (&v)[4]) {
        const Four<AT> a = *reinterpret_cast<const Four<AT> *>(x + e);
        float u[4];
#pragma unroll
        for (int q = 0; q < 4; q++) u[q] = v[q] = to_f32(a.v[q]);
        if (rot.table && e < rot.dims) {
            const float4 cs = *reinterpret_cast<const float4 *>(table + e / 2);
            v[0] = fmaf(u[0], cs.x, -(u[1] * cs.y)), v[1] = fmaf(u[1], cs.x, u[0] * cs.y);
            v[2] = fmaf(u[2], cs.z, -(u[3] * cs.w)), v[3] = fmaf(u[3], cs.z, u[2] * cs.w);
        }
    };
    auto squares = [](const float (&v)[4]) { return fmaf(v[0], v[0], v[1] * v[1]) + fmaf(v[2], v[2], v[3] * v[3]); };
    const int first = 4 * (threadIdx.x & 31);
    float v[4] = {}, w[4];   // the first 128 elements stay in registers
    if (first < dim) four(first, v);
    float ss = squares(v);
#pragma unroll 1
    for (int e = first + 128; e < dim; e += 128) {
        four(e, w);
        ss += squares(w);
    }
    const float r = norm ? 1.0f / sqrtf(warp_sum(ss) / (float)dim + eps) : 1.0f;
    auto scaled = [&](int e, float (&v)[4]) {
#pragma unroll
        for (int q = 0; q < 4; q++) v[q] *= r;
        put(e, v);
    };
    if (first < dim) scaled(first, v);
#pragma unroll 1
    for (int e = first + 128; e < dim; e += 128) {
        four(e, w);
        scaled(e, w);
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
    auto finish = [&](const AT *x, auto *out) {
        typedef typename std::remove_pointer<decltype(out)>::type OT;
        if (a.fours) rotated_normed_fours(x, a.rot, pos, a.dim, a.qk_norm, a.eps, [&](int e, const float (&v)[4]) { store_four(out + e, v); });
        else rotated_normed_row(x, a.rot, pos, a.dim, a.qk_norm, a.eps, [&](int e, float v) { out[e] = from_f32<OT>(v); });
    };
    if (unit < a.heads) {
        finish(reinterpret_cast<const AT *>(a.q) + row + (size_t)unit * a.dim, reinterpret_cast<AT *>(a.qn) + ((size_t)t * a.heads + unit) * a.dim);
    } else if (unit < a.heads + a.kv_heads) {
        const int g = unit - a.heads;
        finish(reinterpret_cast<const AT *>(a.k) + row + (size_t)g * a.dim, reinterpret_cast<CT *>(a.kc) + (slot * a.kv_heads + g) * a.dim);
    } else {
        const int g = unit - a.heads - a.kv_heads;
        const AT *src = reinterpret_cast<const AT *>(a.v) + row + (size_t)g * a.vdim;
        CT *out = reinterpret_cast<CT *>(a.vc) + (slot * a.kv_heads + g) * a.vdim;
        if (a.fours && sizeof(AT) == sizeof(CT) && a.vdim % 4 == 0) {
            for (int e = 4 * lane; e < a.vdim; e += 128) *reinterpret_cast<Four<CT> *>(out + e) = *reinterpret_cast<const Four<CT> *>(src + e);
        } else {
            for (int e = lane; e < a.vdim; e += 32) out[e] = from_f32<CT>(to_f32(src[e]));
        }
    }
}

// A step CTA: 64 keys at a time of one key/value head, for the rep query heads that share it.  bf16 rings with dim % 32 ==
// 0 and vdim % 16 == 0: the products run on tensor cores, the query heads as the 16 rows (queries and weights enter as bf16
// hi + lo parts); else on the CUDA cores.
constexpr int AS_KEYS = 64, AS_THREADS = 256, AS_PE = AS_KEYS + 8;
template <class CT>
struct AttentionStepSmem {
    int kp, vp, rows;                          // elements per staged key / value row; query rows of the products (0: no tensor cores)
    uint32_t k, v, q, s, acc, stat, qh, ph, bytes;   // qh, ph: hi parts, the lo parts behind them
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
    L.rows = sizeof(CT) == 2 && dim % 32 == 0 && vdim % 16 == 0 ? (rep + 15) & ~15 : 0;
    L.qh = (L.stat + (uint32_t)(4 * rep * 4) + 15) & ~15u;
    L.ph = L.qh + (uint32_t)(2 * L.rows * L.kp * 2);
    L.bytes = L.ph + (uint32_t)(2 * L.rows * AS_PE * 2);
    return L;
}
// keys per chunk when n of them are split over at most `chunks` CTAs
__device__ __forceinline__ int attention_chunk_keys(int n, int chunks) { return max(AS_KEYS, ((n + chunks - 1) / chunks + AS_KEYS - 1) / AS_KEYS * AS_KEYS); }

// Block (chunk, g, t) of chunks x kv_heads x tokens.  Waits for the previous launch itself.
template <class AT, class CT>
__device__ __forceinline__ void attention_step_block(const WindowAttentionArgs &a, int chunk, int g, int t, int chunks, uint8_t *as_smem) {
    const int rep = a.heads / a.kv_heads, dim = a.dim, vdim = a.vdim;
    const AttentionStepSmem<CT> L = attention_step_smem<CT>(rep, dim, vdim);
    CT *sk = reinterpret_cast<CT *>(as_smem + L.k), *sv = reinterpret_cast<CT *>(as_smem + L.v);
    float *sq = reinterpret_cast<float *>(as_smem + L.q), *ss = reinterpret_cast<float *>(as_smem + L.s), *acc = reinterpret_cast<float *>(as_smem + L.acc);
    float *s_m = reinterpret_cast<float *>(as_smem + L.stat), *s_l = s_m + rep, *s_c = s_l + rep, *s_g = s_c + rep;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    constexpr int E = 16 / (int)sizeof(CT);
    const bool vec = dim % E == 0 && vdim % E == 0;
    pdl_wait();
    const int pos0 = *a.pos0, pos = pos0 + t;
    const int n = a.window > 0 ? min(pos + 1, a.window) : pos + 1, per = attention_chunk_keys(n, chunks), active = (n + per - 1) / per;
    if (chunk >= active) return;
    const int lo = pos + 1 - n + chunk * per, hi = min(lo + per, pos + 1);
    const int fresh = a.fresh ? pos0 : pos + 1;   // keys from here on come from the projections
    const CT *kc = reinterpret_cast<const CT *>(a.kc) + (size_t)g * dim, *vc = reinterpret_cast<const CT *>(a.vc) + (size_t)g * vdim;
    const size_t ldk = (size_t)a.kv_heads * dim, ldv = (size_t)a.kv_heads * vdim;
    auto load = [&](int base) {
        const int cached = min(min(hi, fresh) - base, AS_KEYS);   // rows that the rings hold
        if (vec) {
            // four threads walk along a key's rows
            const int r = tid >> 2, q0 = tid & 3, key = base + r;
            const bool in = r < cached;
            if (in || key < fresh || key >= hi) {   // else written below
                const size_t slot = (size_t)((in ? key : lo) % a.ring);
                auto row = [&](CT *dst, const CT *src, int n) {
                    for (int c = q0; c < n; c += 4)
                        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst + c * E)), "l"(src + c * E), "r"(in ? 16u : 0u) : "memory");
                };
                row(sk + r * L.kp, kc + slot * ldk, dim / E);
                row(sv + r * L.vp, vc + slot * ldv, vdim / E);
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
            const AT *kx = reinterpret_cast<const AT *>(a.k) + row + (size_t)g * dim;
            if (a.fours)
                rotated_normed_fours(kx, a.rot, key, dim, a.qk_norm, a.eps, [&](int e, const float (&v)[4]) {
                    store_four(sk + r * L.kp + e, v);
                    if (append) store_four(ko + e, v);
                });
            else
                rotated_normed_row(kx, a.rot, key, dim, a.qk_norm, a.eps, [&](int e, float v) {
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
        const AT *qx = reinterpret_cast<const AT *>(a.q) + (size_t)t * a.ld + (size_t)h * dim;
        if (a.fours) rotated_normed_fours(qx, a.rot, pos, dim, a.qk_norm, a.eps, [&](int e, const float (&v)[4]) { store_four(sq + j * dim + e, v); });
        else rotated_normed_row(qx, a.rot, pos, dim, a.qk_norm, a.eps, [&](int e, float v) { sq[j * dim + e] = v; });
        if (lane == 0) {
            s_m[j] = -INFINITY, s_l[j] = 0.f;
            s_g[j] = a.gate ? a.out_mul / (1.0f + expf(-a.gate[(size_t)t * a.ldg + h])) : a.out_mul;
        }
    }
    for (int i = tid; i < rep * vdim; i += AS_THREADS) acc[i] = 0.f;
    bf16 *qhi = reinterpret_cast<bf16 *>(as_smem + L.qh), *qlo = qhi + L.rows * L.kp, *phi = reinterpret_cast<bf16 *>(as_smem + L.ph), *plo = phi + L.rows * AS_PE;
    if (L.rows) {
        __syncthreads();
        for (int i = tid; i < L.rows * dim; i += AS_THREADS) {
            const int j = i / dim, e = i % dim;
            lt_split_store(qhi + j * L.kp + e, qlo + j * L.kp + e, j < rep ? sq[i] : 0.f);
        }
        for (int i = tid; i < (L.rows - rep) * AS_PE; i += AS_THREADS) phi[rep * AS_PE + i] = plo[rep * AS_PE + i] = from_f32<bf16>(0.f);
    }
    const int fg = lane >> 2, tq = lane & 3, mi = lane >> 3, mr = lane & 7;
    const uint32_t a_row = (uint32_t)((mi & 1) * 8 + mr), a_col = (uint32_t)(mi >> 1) * 16u;
    for (int base = lo; base < hi; base += AS_KEYS) {
        const int nk = min(AS_KEYS, hi - base);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        if (L.rows) {   // keys 8 warp .. + 7
            const uint32_t kb = smem_u32(sk) + (uint32_t)((warp * 8 + mr) * L.kp) * 2u + (uint32_t)mi * 16u;
            for (int j0 = 0; j0 < L.rows; j0 += 16) {
                const uint32_t qa = smem_u32(qhi) + ((uint32_t)j0 + a_row) * (uint32_t)L.kp * 2u + a_col, ql = qa + (uint32_t)(L.rows * L.kp) * 2u;
                float c[4][4] = {};
#pragma unroll 2
                for (int k = 0; k < dim / 32; k++) {
                    uint32_t b[4], h0[4], h1[4], l0[4], l1[4];
                    lt_ldmatrix_x4(b, kb + (uint32_t)k * 64u);
                    lt_ldmatrix_x4(h0, qa + (uint32_t)k * 64u);
                    lt_ldmatrix_x4(h1, qa + (uint32_t)k * 64u + 32u);
                    lt_ldmatrix_x4(l0, ql + (uint32_t)k * 64u);
                    lt_ldmatrix_x4(l1, ql + (uint32_t)k * 64u + 32u);
                    lt_mma(c[0], h0, b[0], b[1]);
                    lt_mma(c[1], h1, b[2], b[3]);
                    lt_mma(c[2], l0, b[0], b[1]);
                    lt_mma(c[3], l1, b[2], b[3]);
                }
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const int j = j0 + fg + 8 * (e >> 1), r = warp * 8 + 2 * tq + (e & 1);
                    if (j < rep) ss[j * AS_KEYS + r] = r < nk ? ((c[0][e] + c[1][e]) + (c[2][e] + c[3][e])) * a.scale : -INFINITY;
                }
            }
        } else
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
            if (L.rows) {
                lt_split_store(phi + j * AS_PE + lane, plo + j * AS_PE + lane, p0);
                lt_split_store(phi + j * AS_PE + lane + 32, plo + j * AS_PE + lane + 32, p1);
            } else {
                ss[j * AS_KEYS + lane] = p0;
                ss[j * AS_KEYS + lane + 32] = p1;
            }
            if (lane == 0) {
                const float c = expf(old - m);
                s_c[j] = c;
                s_m[j] = m;
                s_l[j] = fmaf(s_l[j], c, sum);
            }
        }
        __syncthreads();
        const int n4 = (nk + 3) / 4;
        if (L.rows) {   // 16 value columns per warp and pass
            for (int c0 = warp * 16; c0 < vdim; c0 += AS_THREADS / 2)
                for (int j0 = 0; j0 < L.rows; j0 += 16) {
                    const uint32_t pa = smem_u32(phi) + ((uint32_t)j0 + a_row) * (AS_PE * 2) + a_col, pl = pa + (uint32_t)(L.rows * AS_PE) * 2u;
                    const uint32_t vb = smem_u32(sv) + (uint32_t)(((mi & 1) * 8 + mr) * L.vp + c0) * 2u + (uint32_t)(mi >> 1) * 16u;
                    float o[4][4] = {};
#pragma unroll
                    for (int kk = 0; kk < AS_KEYS / 16; kk++) {
                        uint32_t ph[4], pw[4], b[4];
                        lt_ldmatrix_x4(ph, pa + (uint32_t)kk * 32u);
                        lt_ldmatrix_x4(pw, pl + (uint32_t)kk * 32u);
                        lt_ldmatrix_x4_trans(b, vb + (uint32_t)(kk * 16 * L.vp) * 2u);
                        lt_mma(o[0], ph, b[0], b[1]);
                        lt_mma(o[1], ph, b[2], b[3]);
                        lt_mma(o[2], pw, b[0], b[1]);
                        lt_mma(o[3], pw, b[2], b[3]);
                    }
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        const int j = j0 + fg + 8 * (e >> 1);
                        if (j >= rep) continue;
#pragma unroll
                        for (int n = 0; n < 2; n++) {
                            float *to = acc + j * vdim + c0 + n * 8 + 2 * tq + (e & 1);
                            *to = fmaf(*to, s_c[j], o[n][e] + o[n + 2][e]);
                        }
                    }
                }
        } else if (vdim % 2 == 0) {
            for (int i = tid; i < rep * vdim / 2; i += AS_THREADS) {
                const int j = i / (vdim / 2), c = i % (vdim / 2) * 2;
                const float4 *p = reinterpret_cast<const float4 *>(ss + j * AS_KEYS);
                const CT *v = sv + c;
                float o0 = 0.f, o1 = 0.f;
                auto two = [&](int r, float w) {   // rows are padded to 16 bytes: a pair is one access
                    if (E == 8) {
                        const uint32_t x = *reinterpret_cast<const uint32_t *>(v + r * L.vp);
                        o0 = fmaf(w, bf16_lo(x), o0);
                        o1 = fmaf(w, bf16_hi(x), o1);
                    } else {
                        const float2 x = *reinterpret_cast<const float2 *>(v + r * L.vp);
                        o0 = fmaf(w, x.x, o0);
                        o1 = fmaf(w, x.y, o1);
                    }
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
    if (active == 1) {
        for (int i = tid; i < rep * vdim; i += AS_THREADS) {
            const int j = i / vdim, h = g * rep + j;
            act[(size_t)h * vdim + i % vdim] = from_f32<AT>(acc[i] / s_l[j] * s_g[j]);
        }
        return;
    }
    const size_t pl = (size_t)rep * (vdim + 2);
    float *part = a.part + ((size_t)t * a.kv_heads + g) * chunks * pl, *mine = part + (size_t)chunk * pl;
    for (int i = tid; i < rep * vdim; i += AS_THREADS) __stcg(mine + i, acc[i]);
    for (int j = tid; j < rep; j += AS_THREADS) __stcg(mine + rep * vdim + j, s_m[j]), __stcg(mine + rep * (vdim + 1) + j, s_l[j]);
    if (!last_of_head(a.counters + t * a.kv_heads + g, active)) return;
    // the chunks' weights, then their weighted sum; ss is free and holds up to AS_KEYS of them per query head
    for (int j = warp; j < rep; j += AS_THREADS / 32) {
        float mc[2], lc[2], m = -INFINITY, l = 0.f;
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const int c = lane + 32 * i;
            mc[i] = c < active ? __ldcg(part + c * pl + rep * vdim + j) : -INFINITY;
            lc[i] = c < active ? __ldcg(part + c * pl + rep * (vdim + 1) + j) : 0.f;
            m = fmaxf(m, mc[i]);
        }
        m = warp_max(m);
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const float w = expf(mc[i] - m);
            ss[j * AS_KEYS + lane + 32 * i] = w;
            l = fmaf(w, lc[i], l);
        }
        l = warp_sum(l);
        if (lane == 0) s_l[j] = s_g[j] / l;
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

// grid = (chunks, kv_heads, tokens)
template <class AT, class CT>
RNB_GLOBAL void __launch_bounds__(AS_THREADS)
attention_step_kernel(const __grid_constant__ WindowAttentionArgs a) {
    extern __shared__ __align__(16) uint8_t as_smem[];
    pdl_launch_dependents();
    attention_step_block<AT, CT>(a, blockIdx.x, blockIdx.y, blockIdx.z, gridDim.x, as_smem);
}

// Both mixers of a parallel layer, 1..8 tokens, in one launch: n_att = chunks * kv_heads * tokens blocks of attention, then
// heads * n_jb of the delta rule.  Their counters lie apart.
template <class CT, int TI>
RNB_GLOBAL void __launch_bounds__(256)
attention_delta_step_kernel(const __grid_constant__ WindowAttentionArgs a, const __grid_constant__ DeltaArgs d, int chunks, int n_att, int n_jb) {
    extern __shared__ __align__(16) uint8_t ad_smem[];
    pdl_launch_dependents();
    const int b = blockIdx.x;
    if (b < n_att) attention_step_block<float, CT>(a, b % chunks, b / chunks % a.kv_heads, b / chunks / a.kv_heads, chunks, ad_smem);
    else delta_step_block<float, TI>(d, (b - n_att) / n_jb, (b - n_att) % n_jb, n_jb, reinterpret_cast<float *>(ad_smem));
}

}  // namespace rnb
