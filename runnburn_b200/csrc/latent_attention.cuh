// Latent attention: the cache holds one row per position, [latent c (kv_rank) | rotated key part
// (rot_dim)], shared by all heads; the key of head h is [W_uk_h c | rotated part], its value W_uv_h c.
//
// Few tokens (and everything in f32): the absorbed form.  q_h . W_uk_h c = (W_uk_h^T q_h) . c, so the
// query moves into the latent space once (latent_prepare_kernel, which also appends the tokens' cache
// rows), attention runs over the cache rows themselves (latent_attend_kernel, split over the context),
// and the merged latent result is taken to the value space (latent_output_kernel).
// Prompts in bf16: keys and values are expanded by matmuls and latent_prefill_kernel runs causal
// attention on tensor cores.
#pragma once
#include "layer_glue.cuh"

namespace rnb {

struct LatentDims {
    int heads, dim, rot_dim, vdim, rank, ld;   // ld: elements per cache row (kv_rank + rot_dim, padded to 8)
};

// Cache row of one token from its [rank + rot] projection y: c = y / rms(y) * w, rotated key part.
template <class CT>
__device__ __forceinline__ void latent_append_row(const float *y, const float *w, float eps, const LatentDims &d, const Rotation &rot, int pos, CT *cache, float *red) {
    float ss = 0.f;
    for (int i = threadIdx.x; i < d.rank; i += blockDim.x) ss = fmaf(y[i], y[i], ss);
    const float r = 1.0f / sqrtf(block_sum(ss, red) / (float)d.rank + eps);
    CT *row = cache + (size_t)pos * d.ld;
    for (int i = threadIdx.x; i < d.rank; i += blockDim.x) row[i] = from_f32<CT>(y[i] * r * w[i]);
    for (int i = threadIdx.x; i < d.rot_dim; i += blockDim.x)
        row[d.rank + i] = from_f32<CT>(rotated_element(rot, pos, i, [&](int e) { return y[d.rank + e]; }));
}
// grid = tokens
template <class CT>
RNB_GLOBAL void __launch_bounds__(128)
latent_append_kernel(const float *__restrict__ y, const float *__restrict__ w, float eps, const LatentDims d, const Rotation rot, const int *__restrict__ pos0,
                     CT *__restrict__ cache) {
    __shared__ float red[32];
    pdl_launch_dependents();
    pdl_wait();
    latent_append_row<CT>(y + (size_t)blockIdx.x * (d.rank + d.rot_dim), w, eps, d, rot, *pos0 + (int)blockIdx.x, cache, red);
}

// grid = (heads + 1, tokens, ceil(rank / 256)), 128 threads.  Head h: qf[t][h] = [W_uk_h^T q | rotated q];
// the extra column of CTAs appends the token's cache row.  Dynamic shared memory: dim floats.
struct LatentPrepareArgs {
    const float *q, *y, *w;      // [tokens][heads * (dim + rot)], [tokens][rank + rot], [rank]
    const bf16 *uk;              // [heads * dim][rank]
    float *qf;                   // [tokens][heads][rank + rot]
    void *cache;
    const int *pos0;
    float eps;
    LatentDims d;
    Rotation rot;
};
template <class CT>
RNB_GLOBAL void __launch_bounds__(128)
latent_prepare_kernel(const __grid_constant__ LatentPrepareArgs a) {
    extern __shared__ __align__(16) float lp_q[];
    __shared__ float red[32];
    pdl_launch_dependents();
    pdl_wait();
    const LatentDims &d = a.d;
    const int h = blockIdx.x, t = blockIdx.y, pos = *a.pos0 + t, E = d.rank + d.rot_dim;
    if (h == d.heads) {
        if (blockIdx.z == 0)
            latent_append_row<CT>(a.y + (size_t)t * E, a.w, a.eps, d, a.rot, pos, reinterpret_cast<CT *>(a.cache), red);
        return;
    }
    const float *q = a.q + ((size_t)t * d.heads + h) * (d.dim + d.rot_dim);
    float *out = a.qf + ((size_t)t * d.heads + h) * E;
    for (int i = threadIdx.x; i < d.dim; i += 128) lp_q[i] = q[i];
    if (blockIdx.z == 0)
        for (int i = threadIdx.x; i < d.rot_dim; i += 128) out[d.rank + i] = rotated_element(a.rot, pos, i, [&](int e) { return q[d.dim + e]; });
    __syncthreads();
    const int c = blockIdx.z * 256 + 2 * threadIdx.x;
    if (c >= d.rank) return;
    const bf16 *w = a.uk + (size_t)h * d.dim * d.rank + c;
    float s0 = 0.f, s1 = 0.f;
    if (d.rank % 2 == 0) {
#pragma unroll 8
        for (int i = 0; i < d.dim; i++) {
            const uint32_t p = __ldg(reinterpret_cast<const uint32_t *>(w + (size_t)i * d.rank));
            s0 = fmaf(bf16_lo(p), lp_q[i], s0);
            s1 = fmaf(bf16_hi(p), lp_q[i], s1);
        }
        out[c] = s0;
        out[c + 1] = s1;
    } else {
        const bool two = c + 1 < d.rank;
        for (int i = 0; i < d.dim; i++) {
            s0 = fmaf(to_f32(w[(size_t)i * d.rank]), lp_q[i], s0);
            if (two) s1 = fmaf(to_f32(w[(size_t)i * d.rank + 1]), lp_q[i], s1);
        }
        out[c] = s0;
        if (two) out[c + 1] = s1;
    }
}

// Keys [lo, hi) of chunk c when n keys are split over `chunks`.
__device__ __forceinline__ void latent_chunk_range(int n, int chunks, int c, int &lo, int &hi) {
    const int per = (n + chunks - 1) / chunks;
    lo = min(c * per, n);
    hi = min(lo + per, n);
}

// Absorbed attention over one chunk of the cache on the CUDA cores.  grid = (chunks, heads, tokens), 128
// threads; a warp takes every fourth key, lane l elements l + 32 q of a row.  part[t][h][chunk] holds the
// unnormalised latent sum (rank), the maximum and the sum of the weights.
template <class CT, int NQ>
RNB_GLOBAL void __launch_bounds__(128)
latent_attend_kernel(const float *__restrict__ qf, const CT *__restrict__ cache, const LatentDims d, float scale, const int *__restrict__ pos0,
                     float *__restrict__ part) {
    __shared__ float s_o[4][32 * NQ], s_m[4], s_l[4];
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.y, t = blockIdx.z, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, E = d.rank + d.rot_dim;
    int lo, hi;
    latent_chunk_range(*pos0 + t + 1, gridDim.x, blockIdx.x, lo, hi);
    const float *q = qf + ((size_t)t * d.heads + h) * E;
    float qv[NQ], o[NQ], m = -INFINITY, l = 0.f;
#pragma unroll
    for (int i = 0; i < NQ; i++) {
        const int e = lane + 32 * i;
        qv[i] = e < E ? q[e] : 0.f;
        o[i] = 0.f;
    }
    for (int key = lo + warp; key < hi; key += 4) {
        const CT *row = cache + (size_t)key * d.ld;
        float c[NQ], s = 0.f;
#pragma unroll
        for (int i = 0; i < NQ; i++) {
            const int e = lane + 32 * i;
            c[i] = e < E ? to_f32(row[e]) : 0.f;
            s = fmaf(qv[i], c[i], s);
        }
        s = warp_sum(s) * scale;
        const float mn = fmaxf(m, s), corr = expf(m - mn), p = expf(s - mn);
        m = mn;
        l = fmaf(l, corr, p);
#pragma unroll
        for (int i = 0; i < NQ; i++) o[i] = fmaf(p, c[i], o[i] * corr);
    }
#pragma unroll
    for (int i = 0; i < NQ; i++) s_o[warp][lane + 32 * i] = o[i];
    if (lane == 0) s_m[warp] = m, s_l[warp] = l;
    __syncthreads();
    const float M = fmaxf(fmaxf(s_m[0], s_m[1]), fmaxf(s_m[2], s_m[3]));
    float f[4], L = 0.f;
#pragma unroll
    for (int w = 0; w < 4; w++) {
        f[w] = s_m[w] == -INFINITY ? 0.f : expf(s_m[w] - M);
        L = fmaf(f[w], s_l[w], L);
    }
    float *out = part + (((size_t)t * d.heads + h) * gridDim.x + blockIdx.x) * (d.rank + 2);
    for (int e = threadIdx.x; e < d.rank; e += 128) out[e] = f[0] * s_o[0][e] + f[1] * s_o[1][e] + f[2] * s_o[2][e] + f[3] * s_o[3][e];
    if (threadIdx.x == 0) out[d.rank] = M, out[d.rank + 1] = L;
}

// act[t][h * vdim + v] = W_uv_h (merged latent result).  grid = (heads, tokens, row blocks), 128 threads;
// dynamic shared memory rank + chunks floats.
template <class HT>
RNB_GLOBAL void __launch_bounds__(128)
latent_output_kernel(const float *__restrict__ part, const bf16 *__restrict__ uv, const LatentDims d, int chunks, int rows_per_cta, HT *__restrict__ act) {
    extern __shared__ __align__(16) float lo_smem[];
    __shared__ float s_inv;
    pdl_launch_dependents();
    pdl_wait();
    float *ol = lo_smem, *f = lo_smem + d.rank;
    const int h = blockIdx.x, t = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const float *p = part + ((size_t)t * d.heads + h) * chunks * (d.rank + 2);
    if (warp == 0) {
        float M = -INFINITY, L = 0.f;
        for (int c = lane; c < chunks; c += 32) M = fmaxf(M, p[(size_t)c * (d.rank + 2) + d.rank]);
        M = warp_max(M);
        for (int c = lane; c < chunks; c += 32) {
            const float m = p[(size_t)c * (d.rank + 2) + d.rank], e = m == -INFINITY ? 0.f : expf(m - M);
            f[c] = e;
            L = fmaf(e, p[(size_t)c * (d.rank + 2) + d.rank + 1], L);
        }
        L = warp_sum(L);
        if (lane == 0) s_inv = 1.0f / L;
    }
    __syncthreads();
    for (int e = threadIdx.x; e < d.rank; e += 128) {
        float s = 0.f;
#pragma unroll 4
        for (int c = 0; c < chunks; c++) s = fmaf(f[c], p[(size_t)c * (d.rank + 2) + e], s);
        ol[e] = s * s_inv;
    }
    __syncthreads();
    const int v0 = blockIdx.z * rows_per_cta, v1 = min(v0 + rows_per_cta, d.vdim);
    for (int v = v0 + warp; v < v1; v += 4) {
        const bf16 *w = uv + ((size_t)h * d.vdim + v) * d.rank;
        float s = 0.f;
        if (d.rank % 8 == 0) {
            for (int e = lane * 8; e < d.rank; e += 256) {
                const uint4 b = ldg_nc_u4(w + e);
                const uint32_t q[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    s = fmaf(bf16_lo(q[i]), ol[e + 2 * i], s);
                    s = fmaf(bf16_hi(q[i]), ol[e + 2 * i + 1], s);
                }
            }
        } else {
            for (int e = lane; e < d.rank; e += 32) s = fmaf(to_f32(w[e]), ol[e], s);
        }
        s = warp_sum(s);
        if (lane == 0) act[((size_t)t * d.heads + h) * d.vdim + v] = from_f32<HT>(s);
    }
}

// ---- prompts: causal attention over expanded keys and values on tensor cores ---------------------
__device__ __forceinline__ void la_ldmatrix_x4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void la_ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void la_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// (x, y) as packed bf16 plus what the rounding left over, again in bf16
__device__ __forceinline__ void la_split(float x, float y, uint32_t &hi, uint32_t &lo) {
    hi = pg_pack_bf16(x, y);
    lo = pg_pack_bf16(x - bf16_lo(hi), y - bf16_hi(hi));
}

constexpr int LA_ROWS = 128, LA_KEYS = 64, LA_THREADS = 256;
__host__ __device__ inline int la_pad16(int n) { return (n + 15) & ~15; }
__host__ inline size_t latent_prefill_smem(const LatentDims &d, int dvp) {
    return 2 * ((size_t)(LA_ROWS + 2 * LA_KEYS) * (la_pad16(d.dim + d.rot_dim) + 8) + (size_t)2 * LA_KEYS * (dvp + 8));
}
struct LatentPrefillArgs {
    const bf16 *q, *kn, *kr, *v;   // [tokens][heads][dim + rot] (rotated), [keys][heads][dim], cache + rank, [keys][heads][vdim]
    bf16 *act;                     // [tokens][heads * vdim]
    const int *pos0;
    float scale;
    int tokens, vec;               // vec: every row piece is 16-byte aligned and a multiple of 8 elements
    LatentDims d;
};
// grid = (ceil(tokens / 128), heads), 256 threads; warp w owns queries 16w .. 16w + 15 of the CTA's 128.
// Keys come in tiles of 64, double-buffered; the weights enter the value product as bf16 hi + lo parts.
// DVJ: 8-column tiles of the value dimension (vdim <= 8 DVJ).
template <int DVJ>
RNB_GLOBAL void __launch_bounds__(LA_THREADS, 1)
latent_prefill_kernel(const __grid_constant__ LatentPrefillArgs a) {
    extern __shared__ __align__(128) uint8_t la_smem[];
    pdl_launch_dependents();
    pdl_wait();
    const LatentDims &d = a.d;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y;
    const int dk = d.dim + d.rot_dim, dkp = la_pad16(dk), KS = dkp / 16;
    constexpr int DVP = 8 * DVJ;
    const uint32_t kpitch = (uint32_t)(dkp + 8) * 2, vpitch = (uint32_t)(DVP + 8) * 2;
    bf16 *qs = reinterpret_cast<bf16 *>(la_smem);
    bf16 *ks = qs + (size_t)LA_ROWS * (dkp + 8), *vs = ks + (size_t)2 * LA_KEYS * (dkp + 8);
    const uint32_t q_base = smem_u32(qs), k_base = smem_u32(ks), v_base = smem_u32(vs);
    const int i0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * LA_ROWS;   // long rows first
    const int pos0 = *a.pos0, kv_len = pos0 + a.tokens;
    const int n_keys = min(kv_len, pos0 + i0 + LA_ROWS), n_tiles = (n_keys + LA_KEYS - 1) / LA_KEYS;
    const bf16 zero = from_f32<bf16>(0.f);
    // queries, and zeros in the padding columns of every buffer (the copies below never touch those)
    for (int i = tid; i < LA_ROWS * (dkp + 8); i += LA_THREADS) {
        const int r = i / (dkp + 8), c = i % (dkp + 8);
        qs[i] = c < dk && i0 + r < a.tokens ? a.q[((size_t)(i0 + r) * d.heads + h) * dk + c] : zero;
    }
    if (dkp > dk)
        for (int i = tid; i < 2 * LA_KEYS * (dkp - dk); i += LA_THREADS) ks[(size_t)(i / (dkp - dk)) * (dkp + 8) + dk + i % (dkp - dk)] = zero;
    if (DVP > d.vdim)
        for (int i = tid; i < 2 * LA_KEYS * (DVP - d.vdim); i += LA_THREADS) vs[(size_t)(i / (DVP - d.vdim)) * (DVP + 8) + d.vdim + i % (DVP - d.vdim)] = zero;
    auto load_tile = [&](int t) {
        const int st = t & 1, key0 = t * LA_KEYS;
        if (a.vec) {
            const int cn = d.dim / 8, cr = d.rot_dim / 8, cv = d.vdim / 8, per = cn + cr + cv;
            for (int i = tid; i < LA_KEYS * per; i += LA_THREADS) {
                const int r = i / per, c = i % per, key = key0 + r, kk = min(key, kv_len - 1);
                const bf16 *src;
                uint32_t dst;
                if (c < cn) {
                    src = a.kn + ((size_t)kk * d.heads + h) * d.dim + c * 8;
                    dst = k_base + (uint32_t)(st * LA_KEYS + r) * kpitch + (uint32_t)c * 16u;
                } else if (c < cn + cr) {
                    src = a.kr + (size_t)kk * d.ld + (c - cn) * 8;
                    dst = k_base + (uint32_t)(st * LA_KEYS + r) * kpitch + (uint32_t)c * 16u;
                } else {
                    src = a.v + ((size_t)kk * d.heads + h) * d.vdim + (c - cn - cr) * 8;
                    dst = v_base + (uint32_t)(st * LA_KEYS + r) * vpitch + (uint32_t)(c - cn - cr) * 16u;
                }
                const uint32_t nbytes = key < kv_len ? 16u : 0u;
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(nbytes) : "memory");
            }
        } else {
            const int per = dk + d.vdim;
            for (int i = tid; i < LA_KEYS * per; i += LA_THREADS) {
                const int r = i / per, c = i % per, key = key0 + r;
                const bool in = key < kv_len;
                if (c < dk)
                    ks[(size_t)(st * LA_KEYS + r) * (dkp + 8) + c] =
                        !in ? zero : c < d.dim ? a.kn[((size_t)key * d.heads + h) * d.dim + c] : a.kr[(size_t)key * d.ld + c - d.dim];
                else
                    vs[(size_t)(st * LA_KEYS + r) * (DVP + 8) + c - dk] = in ? a.v[((size_t)key * d.heads + h) * d.vdim + c - dk] : zero;
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load_tile(0);
    const int g = lane >> 2, tq = lane & 3, mi = lane >> 3, mr = lane & 7;
    int qi[2], pos[2];
    bool live[2];
#pragma unroll
    for (int e = 0; e < 2; e++) {
        qi[e] = i0 + warp * 16 + g + 8 * e;
        live[e] = qi[e] < a.tokens;
        pos[e] = live[e] ? pos0 + qi[e] : kv_len - 1;   // rows past the end see everything and are never stored
    }
    float o[DVJ][4], m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
#pragma unroll
    for (int j = 0; j < DVJ; j++) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
    const float sl2 = a.scale * 1.4426950408889634f;
    // A fragments: matrices (rows 0-7, k 0-7), (rows 8-15, k 0-7), (rows 0-7, k 8-15), (rows 8-15, k 8-15)
    const uint32_t q_addr = q_base + (uint32_t)(warp * 16 + (mi & 1) * 8 + mr) * kpitch + (uint32_t)(mi >> 1) * 16u;
    for (int t = 0; t < n_tiles; t++) {
        if (t + 1 < n_tiles) {
            load_tile(t + 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const uint32_t k_st = k_base + (uint32_t)(t & 1) * LA_KEYS * kpitch, v_st = v_base + (uint32_t)(t & 1) * LA_KEYS * vpitch;
        float s[8][4];
#pragma unroll
        for (int j = 0; j < 8; j++) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
        // B fragments of two key tiles per ldmatrix: (keys 0-7, k 0-7), (keys 0-7, k 8-15), (keys 8-15, k 0-7), (keys 8-15, k 8-15)
        const uint32_t kb = k_st + (uint32_t)((mi >> 1) * 8 + mr) * kpitch + (uint32_t)(mi & 1) * 16u;
        for (int kk = 0; kk < KS; kk++) {
            uint32_t af[4];
            la_ldmatrix_x4(af, q_addr + (uint32_t)kk * 32u);
#pragma unroll
            for (int jp = 0; jp < 4; jp++) {
                uint32_t b[4];
                la_ldmatrix_x4(b, kb + (uint32_t)(jp * 16) * kpitch + (uint32_t)kk * 32u);
                la_mma(s[2 * jp], af, b[0], b[1]);
                la_mma(s[2 * jp + 1], af, b[2], b[3]);
            }
        }
        const int key0 = t * LA_KEYS + 2 * tq;
        const bool need_mask = t * LA_KEYS + LA_KEYS - 1 > min(pos[0], pos[1]);
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int j = 0; j < 8; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                float x = s[j][e] * sl2;
                if (need_mask && key0 + j * 8 + (e & 1) > pos[e >> 1]) x = -INFINITY;
                s[j][e] = x;
                mx[e >> 1] = fmaxf(mx[e >> 1], x);
            }
        float corr[2], m_use[2], rs[2] = {0.f, 0.f};
#pragma unroll
        for (int e = 0; e < 2; e++) {
            mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 1));
            mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 2));
            const float mn = fmaxf(m_run[e], mx[e]);
            m_use[e] = mn == -INFINITY ? 0.f : mn;
            corr[e] = exp2f(m_run[e] - m_use[e]);
            m_run[e] = mn;
        }
        uint32_t ph[4][4], pl[4][4];
#pragma unroll
        for (int j = 0; j < 8; j++) {
            const float p0 = exp2f(s[j][0] - m_use[0]), p1 = exp2f(s[j][1] - m_use[0]);
            const float p2 = exp2f(s[j][2] - m_use[1]), p3 = exp2f(s[j][3] - m_use[1]);
            rs[0] += p0 + p1;
            rs[1] += p2 + p3;
            la_split(p0, p1, ph[j >> 1][2 * (j & 1)], pl[j >> 1][2 * (j & 1)]);
            la_split(p2, p3, ph[j >> 1][2 * (j & 1) + 1], pl[j >> 1][2 * (j & 1) + 1]);
        }
#pragma unroll
        for (int e = 0; e < 2; e++) {
            rs[e] += __shfl_xor_sync(0xffffffffu, rs[e], 1);
            rs[e] += __shfl_xor_sync(0xffffffffu, rs[e], 2);
            l_run[e] = fmaf(l_run[e], corr[e], rs[e]);
        }
#pragma unroll
        for (int j = 0; j < DVJ; j++) {
            o[j][0] *= corr[0];
            o[j][1] *= corr[0];
            o[j][2] *= corr[1];
            o[j][3] *= corr[1];
        }
#pragma unroll
        for (int kk = 0; kk < 4; kk++) {
            const uint32_t vb = v_st + (uint32_t)(kk * 16 + (mi & 1) * 8 + mr) * vpitch + (uint32_t)(mi >> 1) * 16u;
#pragma unroll
            for (int jp = 0; jp < DVJ / 2; jp++) {
                uint32_t b[4];
                la_ldmatrix_x4_trans(b, vb + (uint32_t)jp * 32u);
                la_mma(o[2 * jp], ph[kk], b[0], b[1]);
                la_mma(o[2 * jp], pl[kk], b[0], b[1]);
                la_mma(o[2 * jp + 1], ph[kk], b[2], b[3]);
                la_mma(o[2 * jp + 1], pl[kk], b[2], b[3]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int e = 0; e < 2; e++) {
        if (!live[e]) continue;
        const float inv = 1.0f / l_run[e];
        bf16 *dst = a.act + ((size_t)qi[e] * d.heads + h) * d.vdim;
#pragma unroll
        for (int j = 0; j < DVJ; j++)
#pragma unroll
            for (int x = 0; x < 2; x++)
                if (8 * j + 2 * tq + x < d.vdim) dst[8 * j + 2 * tq + x] = from_f32<bf16>(o[j][2 * e + x] * inv);
    }
}

}  // namespace rnb
