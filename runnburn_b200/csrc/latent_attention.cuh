// Latent attention: the cache holds one row per position, [latent c (kv_rank) | rotated key part
// (rot_dim)], shared by all heads; the key of head h is [W_uk_h c | rotated part], its value W_uv_h c.
//
// Few tokens (and everything in f32): the absorbed form.  q_h . W_uk_h c = (W_uk_h^T q_h) . c, so the
// query moves into the latent space once (latent_prepare_kernel, which also appends the tokens' cache
// rows), attention runs over the cache rows themselves (latent_attend_kernel, split over the context),
// and the merged latent result is taken to the value space (latent_output_kernel).
// Prompts in bf16: keys and values are expanded by matmuls and causal_attention_kernel runs over them.
#pragma once
#include "causal_attention.cuh"

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

// grid = (heads + 1, tokens, ceil(rank / 128)), 512 threads.  Head h: qf[t][h] = [W_uk_h^T q | rotated q];
// the extra column of CTAs appends the token's cache row.  16 threads hold 8 columns each, 32 groups of them
// share the key dimensions; the first rows of W_uk are loaded ahead of the dependency wait.
// Dynamic shared memory: dim + 32 * 128 floats.
struct LatentPrepareArgs {
    const float *q, *y, *w;      // [tokens][heads * (dim + rot)], [tokens][rank + rot], [rank]
    const bf16 *uk;              // [heads * dim][rank]
    void *qf;                    // [tokens][heads][qld] of QT, zeros from rank + rot on
    int qld;
    void *cache;
    const int *pos0;
    float eps;
    LatentDims d;
    Rotation rot;
};
constexpr int LP_THREADS = 512, LP_COLS = 128, LP_GROUPS = LP_THREADS / (LP_COLS / 8), LP_BATCH = 4;
template <class CT, class QT>
RNB_GLOBAL void __launch_bounds__(LP_THREADS)
latent_prepare_kernel(const __grid_constant__ LatentPrepareArgs a) {
    extern __shared__ __align__(16) float lp_smem[];
    __shared__ float red[32];
    pdl_launch_dependents();
    const LatentDims &d = a.d;
    const int h = blockIdx.x, t = blockIdx.y, E = d.rank + d.rot_dim, tid = threadIdx.x;
    if (h == d.heads) {
        pdl_wait();
        if (blockIdx.z == 0)
            latent_append_row<CT>(a.y + (size_t)t * E, a.w, a.eps, d, a.rot, *a.pos0 + t, reinterpret_cast<CT *>(a.cache), red);
        return;
    }
    float *sq = lp_smem, *sr = lp_smem + ((d.dim + 3) & ~3);
    const int grp = tid / (LP_COLS / 8), cl = tid % (LP_COLS / 8) * 8, c = blockIdx.z * LP_COLS + cl;
    const bool vec = d.rank % 8 == 0, in = c < d.rank;
    const bf16 *w = a.uk + (size_t)h * d.dim * d.rank + c;
    uint4 b[LP_BATCH];
    auto fetch = [&](int i0) {
#pragma unroll
        for (int k = 0; k < LP_BATCH; k++) {
            const int i = i0 + LP_GROUPS * k + grp;
            b[k] = vec && in && i < d.dim ? ldg_nc_u4(w + (size_t)i * d.rank) : make_uint4(0u, 0u, 0u, 0u);
        }
    };
    fetch(0);
    pdl_wait();
    const float *q = a.q + ((size_t)t * d.heads + h) * (d.dim + d.rot_dim);
    QT *out = reinterpret_cast<QT *>(a.qf) + ((size_t)t * d.heads + h) * a.qld;
    for (int i = tid; i < d.dim; i += LP_THREADS) sq[i] = q[i];
    if (blockIdx.z == 0)
        for (int i = tid; i < a.qld - d.rank; i += LP_THREADS)
            out[d.rank + i] = from_f32<QT>(i < d.rot_dim ? rotated_element(a.rot, *a.pos0 + t, i, [&](int e) { return q[d.dim + e]; }) : 0.f);
    __syncthreads();
    if (!vec) {
        for (int e = blockIdx.z * LP_COLS + tid; e < min(d.rank, (int)(blockIdx.z + 1) * LP_COLS); e += LP_THREADS) {
            const bf16 *col = a.uk + (size_t)h * d.dim * d.rank + e;
            float s = 0.f;
            for (int i = 0; i < d.dim; i++) s = fmaf(to_f32(col[(size_t)i * d.rank]), sq[i], s);
            out[e] = from_f32<QT>(s);
        }
        return;
    }
    float acc[8] = {};
    for (int i0 = 0; i0 < d.dim; i0 += LP_GROUPS * LP_BATCH) {
        if (i0) fetch(i0);
#pragma unroll
        for (int k = 0; k < LP_BATCH; k++) {
            const int i = i0 + LP_GROUPS * k + grp;
            const float qv = i < d.dim ? sq[i] : 0.f;
            const uint32_t p[4] = {b[k].x, b[k].y, b[k].z, b[k].w};
#pragma unroll
            for (int e = 0; e < 4; e++) {
                acc[2 * e] = fmaf(bf16_lo(p[e]), qv, acc[2 * e]);
                acc[2 * e + 1] = fmaf(bf16_hi(p[e]), qv, acc[2 * e + 1]);
            }
        }
    }
#pragma unroll
    for (int e = 0; e < 8; e++) sr[grp * LP_COLS + cl + e] = acc[e];
    __syncthreads();
    const int e = blockIdx.z * LP_COLS + tid;
    if (tid < LP_COLS && e < d.rank) {
        float s = 0.f;
#pragma unroll 8
        for (int k = 0; k < LP_GROUPS; k++) s += sr[k * LP_COLS + tid];
        out[e] = from_f32<QT>(s);
    }
}

// n keys split over at most `chunks` CTAs: at least 128 keys each (a shorter chunk costs more in merging than it
// saves), in whole units of 32.
__device__ __forceinline__ int latent_chunk_keys(int n, int chunks) { return max(128, ((n + chunks - 1) / chunks + 31) & ~31); }
__device__ __forceinline__ void latent_chunk_range(int n, int chunks, int c, int &lo, int &hi) {
    const int per = latent_chunk_keys(n, chunks);
    lo = min(c * per, n);
    hi = min(lo + per, n);
}

__host__ __device__ __forceinline__ int latent_part_ld(int rank) { return ((rank + 3) & ~3) + 4; }

// Absorbed attention over one chunk of the cache on the CUDA cores.  grid = (chunks, heads, tokens), 128
// threads; a warp takes every fourth key, lane l elements l + 32 q of a row.  part[t][h][chunk] (latent_part_ld
// floats) holds the unnormalised latent sum (rank), the maximum and the sum of the weights.
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
    if (lo == hi) return;   // the merge knows how many chunks hold keys
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
    float *out = part + (((size_t)t * d.heads + h) * gridDim.x + blockIdx.x) * latent_part_ld(d.rank);
    for (int e = threadIdx.x; e < d.rank; e += 128) out[e] = f[0] * s_o[0][e] + f[1] * s_o[1][e] + f[2] * s_o[2][e] + f[3] * s_o[3][e];
    if (threadIdx.x == 0) out[d.rank] = M, out[d.rank + 1] = L;
}

// act[t * lda + h * vdim + v] = mul * W_uv_h (merged latent result).  grid = (heads, tokens, row blocks), 512 threads: four
// groups of 128 share the chunks, 16 warps share the rows.  Dynamic shared memory 5 * rank4 + max_chunks floats.
constexpr int LO_THREADS = 512;
template <class HT>
RNB_GLOBAL void __launch_bounds__(LO_THREADS)
latent_output_kernel(const float *__restrict__ part, const bf16 *__restrict__ uv, const LatentDims d, int max_chunks, const int *__restrict__ pos0, int rows_per_cta,
                     HT *__restrict__ act, int lda, float mul) {
    extern __shared__ __align__(16) float lo_smem[];
    __shared__ float s_inv;
    pdl_launch_dependents();
    const int h = blockIdx.x, t = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, R4 = (d.rank + 3) & ~3, ld = latent_part_ld(d.rank);
    const int v0 = blockIdx.z * rows_per_cta, v1 = min(v0 + rows_per_cta, d.vdim);
    if (gridDim.y == 1) prefetch_l2(uv + ((size_t)h * d.vdim + v0) * d.rank, (size_t)(v1 - v0) * d.rank * 2, threadIdx.x, LO_THREADS);
    pdl_wait();
    float *ol = lo_smem, *grp = lo_smem + R4, *f = grp + 4 * R4;
    const float *p = part + ((size_t)t * d.heads + h) * max_chunks * ld;
    const int keys = *pos0 + t + 1, per = latent_chunk_keys(keys, max_chunks), chunks = (keys + per - 1) / per;
    if (warp == 0) {
        float M = -INFINITY, L = 0.f;
        for (int c = lane; c < chunks; c += 32) M = fmaxf(M, p[(size_t)c * ld + d.rank]);
        M = warp_max(M);
        for (int c = lane; c < chunks; c += 32) {
            const float m = p[(size_t)c * ld + d.rank], e = m == -INFINITY ? 0.f : expf(m - M);
            f[c] = e;
            L = fmaf(e, p[(size_t)c * ld + d.rank + 1], L);
        }
        L = warp_sum(L);
        if (lane == 0) s_inv = 1.0f / L;
    }
    __syncthreads();
    const int q = threadIdx.x >> 7;
    for (int e = (threadIdx.x & 127) * 4; e < R4; e += 512) {
        float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
        for (int c = q; c < chunks; c += 4) {
            const float4 x = *reinterpret_cast<const float4 *>(p + (size_t)c * ld + e);
            const float w = f[c];
            if (w != 0.f) s.x = fmaf(w, x.x, s.x), s.y = fmaf(w, x.y, s.y), s.z = fmaf(w, x.z, s.z), s.w = fmaf(w, x.w, s.w);
        }
        *reinterpret_cast<float4 *>(grp + q * R4 + e) = s;
    }
    __syncthreads();
    for (int e = threadIdx.x; e < d.rank; e += LO_THREADS) ol[e] = (grp[e] + grp[R4 + e] + grp[2 * R4 + e] + grp[3 * R4 + e]) * s_inv;
    __syncthreads();
    for (int v = v0 + warp; v < v1; v += LO_THREADS / 32) {
        const bf16 *w = uv + ((size_t)h * d.vdim + v) * d.rank;
        float s = 0.f;
        if (d.rank % 8 == 0) {
#pragma unroll 2
            for (int e = lane * 8; e < d.rank; e += 256) {
                const uint4 b = ldg_nc_u4(w + e);
                const uint32_t x[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    s = fmaf(bf16_lo(x[i]), ol[e + 2 * i], s);
                    s = fmaf(bf16_hi(x[i]), ol[e + 2 * i + 1], s);
                }
            }
        } else {
            for (int e = lane; e < d.rank; e += 32) s = fmaf(to_f32(w[e]), ol[e], s);
        }
        s = warp_sum(s);
        if (lane == 0) act[(size_t)t * lda + h * d.vdim + v] = from_f32<HT>(s * mul);
    }
}

// ---- the same over a bf16 cache on tensor cores ---------------------------------------------------
// The 16 rows of the products are 16 heads (they share every cache row).  Tiles of 64 keys, two stages;
// 8 warps: scores of 8 keys each, then 1/8 of the latent columns each (8 NT per warp).  The query enters in
// bf16, the weights as bf16 hi + lo parts.  grid = (chunks, ceil(heads / 16), tokens); rank and cache rows
// multiples of 8.
constexpr int LM_KEYS = 64, LM_THREADS = 256;
struct LatentMmaSmem {
    uint32_t pitch, q, s, phi, plo, stat, bytes;
};
__host__ __device__ inline LatentMmaSmem latent_mma_smem(const LatentDims &d) {
    LatentMmaSmem L;
    const uint32_t ep = (uint32_t)((d.rank + d.rot_dim + 31) & ~31);   // two k-steps per B load
    L.pitch = (ep + 8) * 2;
    L.q = 2 * LM_KEYS * L.pitch;
    L.s = L.q + 16 * L.pitch;
    L.phi = L.s + 16 * (LM_KEYS + 4) * 4;
    L.plo = L.phi + 16 * (LM_KEYS + 8) * 2;
    L.stat = L.plo + 16 * (LM_KEYS + 8) * 2;
    L.bytes = L.stat + 3 * 16 * 4;
    return L;
}
template <int NT>
RNB_GLOBAL void __launch_bounds__(LM_THREADS)
latent_attend_mma_kernel(const bf16 *__restrict__ qf, const bf16 *__restrict__ cache, const LatentDims d, float scale, const int *__restrict__ pos0,
                         float *__restrict__ part) {
    extern __shared__ __align__(128) uint8_t lm_smem[];
    pdl_launch_dependents();
    pdl_wait();
    const LatentMmaSmem L = latent_mma_smem(d);
    const uint32_t base = smem_u32(lm_smem);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h0 = blockIdx.y * 16, t = blockIdx.z, E = d.rank + d.rot_dim;
    const int EP = (int)(L.pitch / 2) - 8, ld = latent_part_ld(d.rank);
    int lo, hi;
    latent_chunk_range(*pos0 + t + 1, gridDim.x, blockIdx.x, lo, hi);
    if (lo == hi) return;
    float *ss = reinterpret_cast<float *>(lm_smem + L.s), *s_m = reinterpret_cast<float *>(lm_smem + L.stat), *s_l = s_m + 16, *s_c = s_l + 16;
    bf16 *phi = reinterpret_cast<bf16 *>(lm_smem + L.phi), *plo = reinterpret_cast<bf16 *>(lm_smem + L.plo);
    constexpr int PE = LM_KEYS + 8, SE = LM_KEYS + 4;
    auto load_tile = [&](int i) {
        const uint32_t st = base + (uint32_t)(i & 1) * LM_KEYS * L.pitch;
        const int r = tid >> 2, key = lo + i * LM_KEYS + r;   // four threads walk along a row
        for (int q = tid & 3; q < EP / 8; q += 4) {
            // the row's padding (up to ld) is never written by an append; what lies past E meets zero query columns, so it
            // only has to be finite: it is taken as zero
            const bool in = key < hi && q * 8 < E;
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(st + (uint32_t)r * L.pitch + (uint32_t)q * 16u),
                         "l"(cache + (size_t)min(key, hi - 1) * d.ld + min(q * 8, d.ld - 8)), "r"(in ? (uint32_t)min(16, (E - q * 8) * 2) : 0u)
                         : "memory");
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    const int n_tiles = (hi - lo + LM_KEYS - 1) / LM_KEYS;
    if (n_tiles > 0) {
        // query rows (pitch EP in memory), part of the first tile's copy group
        const int r = tid >> 4;
        for (int q = tid & 15; q < EP / 8; q += 16) {
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(base + L.q + (uint32_t)r * L.pitch + (uint32_t)q * 16u),
                         "l"(qf + ((size_t)t * d.heads + min(h0 + r, d.heads - 1)) * EP + q * 8), "r"(h0 + r < d.heads ? 16u : 0u)
                         : "memory");
        }
        load_tile(0);
    }
    if (tid < 16) s_m[tid] = -INFINITY, s_l[tid] = 0.f;
    float o[NT][4];
#pragma unroll
    for (int n = 0; n < NT; n++) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
    const int g = lane >> 2, tq = lane & 3, mi = lane >> 3, mr = lane & 7, c0 = warp * 8 * NT;
    const uint32_t a_off = (uint32_t)((mi & 1) * 8 + mr), a_col = (uint32_t)(mi >> 1) * 16u;
    for (int it = 0; it < n_tiles; it++) {
        if (it + 1 < n_tiles) {
            load_tile(it + 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const uint32_t st = base + (uint32_t)(it & 1) * LM_KEYS * L.pitch;
        {   // scores of keys 8 warp .. + 7; independent accumulators hide the MMA latency
            float s[4][4] = {};
            const uint32_t qa = base + L.q + a_off * L.pitch + a_col, ka = st + (uint32_t)(warp * 8 + mr) * L.pitch + (uint32_t)mi * 16u;
#pragma unroll 2
            for (int k = 0; k < EP / 32; k++) {
                uint32_t b[4], a0[4], a1[4];
                lt_ldmatrix_x4(b, ka + (uint32_t)k * 64u);
                lt_ldmatrix_x4(a0, qa + (uint32_t)k * 64u);
                lt_ldmatrix_x4(a1, qa + (uint32_t)k * 64u + 32u);
                lt_mma(s[2 * (k & 1)], a0, b[0], b[1]);
                lt_mma(s[2 * (k & 1) + 1], a1, b[2], b[3]);
            }
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int key = lo + it * LM_KEYS + warp * 8 + 2 * tq + (e & 1);
                const float v = (s[0][e] + s[1][e]) + (s[2][e] + s[3][e]);
                ss[(g + 8 * (e >> 1)) * SE + warp * 8 + 2 * tq + (e & 1)] = key < hi ? v * scale : -INFINITY;
            }
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 2; i++) {   // softmax bookkeeping of heads 2 warp, 2 warp + 1
            const int r = 2 * warp + i;
            const float x0 = ss[r * SE + lane], x1 = ss[r * SE + lane + 32], m_old = s_m[r];
            const float m = fmaxf(m_old, warp_max(fmaxf(x0, x1)));
            const float p0 = expf(x0 - m), p1 = expf(x1 - m), sum = warp_sum(p0 + p1);
            lt_split_store(phi + r * PE + lane, plo + r * PE + lane, p0);
            lt_split_store(phi + r * PE + lane + 32, plo + r * PE + lane + 32, p1);
            if (lane == 0) {
                const float c = expf(m_old - m);
                s_c[r] = c;
                s_m[r] = m;
                s_l[r] = fmaf(s_l[r], c, sum);
            }
        }
        __syncthreads();
        const float c_lo = s_c[g], c_hi = s_c[g + 8];
#pragma unroll
        for (int n = 0; n < NT; n++) {
            o[n][0] *= c_lo;
            o[n][1] *= c_lo;
            o[n][2] *= c_hi;
            o[n][3] *= c_hi;
        }
#pragma unroll
        for (int kk = 0; kk < LM_KEYS / 16; kk++) {
            uint32_t ah[4], al[4];
            const uint32_t pa = a_off * (PE * 2) + (uint32_t)kk * 32u + a_col;
            lt_ldmatrix_x4(ah, base + L.phi + pa);
            lt_ldmatrix_x4(al, base + L.plo + pa);
            const uint32_t va = st + (uint32_t)(kk * 16 + (mi & 1) * 8 + mr) * L.pitch + (uint32_t)(mi >> 1) * 16u + (uint32_t)c0 * 2u;
#pragma unroll
            for (int np = 0; np < (NT + 1) / 2; np++) {
                if (c0 + np * 16 >= EP) break;
                uint32_t b[4];
                lt_ldmatrix_x4_trans(b, va + (uint32_t)np * 32u);
                lt_mma(o[2 * np], ah, b[0], b[1]);
                lt_mma(o[2 * np], al, b[0], b[1]);
                if (2 * np + 1 < NT) {
                    lt_mma(o[2 * np + 1], ah, b[2], b[3]);
                    lt_mma(o[2 * np + 1], al, b[2], b[3]);
                }
            }
        }
        __syncthreads();
    }
    __syncthreads();
    float *out = part + (((size_t)t * d.heads + h0) * gridDim.x + blockIdx.x) * ld;
    const size_t hs = (size_t)gridDim.x * ld;
#pragma unroll
    for (int n = 0; n < NT; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int r = g + 8 * (e >> 1), c = c0 + n * 8 + 2 * tq + (e & 1);
            if (h0 + r < d.heads && c < d.rank) out[r * hs + c] = o[n][e];
        }
    if (tid < 16 && h0 + tid < d.heads) {
        out[tid * hs + d.rank] = s_m[tid];
        out[tid * hs + d.rank + 1] = s_l[tid];
    }
}

}  // namespace rnb
