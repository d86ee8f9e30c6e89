// Gated delta rule: a matrix state per head that decays as a whole and is corrected towards v at key k,
//   S <- g S,   u = beta (v - S^T k),   S <- S + k u^T,   o = S^T q
// with g = exp(-exp(A) softplus(a + dt)) and beta = sigmoid(b) per head and token, q and k unit vectors shared by
// heads / kv_heads heads, q, k and v each behind a short causal convolution per channel and silu.  State
// [heads][dim][vdim] f32; the projections of the last tokens wait in a ring for the convolutions of the next
// call ([DR_RING(taps)][channels], position p in row p % rows; positions before 0 are zeros).
//
//   delta_step_kernel      token by token: 1..8 tokens in one launch with head norm and gate; also prompts in f32 or odd sizes
//   delta_prepare_kernel   prompts in bf16, all 16-token tiles at once: convolutions, norms, and per tile and head
//                          the 16 x 16 matrices that turn a state into the tile's corrections and outputs
//   delta_tile_kernel      walks the tiles of a head in order on tensor cores, the state in f32 accumulators
//
// Within a tile, with G_ts = g_{s+1} .. g_t, raw (unnormalised) keys y and queries x, and their inverse norms a, b:
//   (I + M) U = beta (V - (G_t0 a_t y_t) S0),   M_ts = beta_t G_ts a_t a_s (y_t . y_s) for s < t
//   o_t = b_t (G_t0 x_t S0 + sum_{s <= t} G_ts a_s (x_t . y_s) u_s),   S = G_T0 S0 + sum_s G_Ts a_s y_s u_s^T
// G is summed in logarithms pair by pair and never divided.
#pragma once
#include "linear_state.cuh"
#include "mma_bf16.cuh"

namespace rnb {

constexpr float DR_UNIT_EPS = 1e-6f;
constexpr int DR_BLOCK = 8;                                      // tokens that a step kernel stages at a time
__host__ __device__ inline int delta_ring_rows(int taps) { return taps - 1 + DR_BLOCK; }
__device__ __forceinline__ float softplus_f32(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float sigmoid_f32(float x) { return 1.0f / (1.0f + expf(-x)); }

struct DeltaArgs {
    const void *p;             // projections (AT), token t at p + t * ld: q [kv_heads * dim] at 0, k, v [heads * vdim], g at the offsets below
    const float *ba;           // [tokens][ld_ba]: b [heads], then a [heads] at a_at
    const float *conv;         // [taps][channels]: q, k and v channels one after the other, the last row for the current input
    const float *a_log, *dt;   // [heads]
    const float *norm;         // step: [vdim]
    float *ring, *state;
    float *o, *act;            // o [tokens][heads][vdim]; act: rows of lda, null: o only
    int *counters;             // [heads], zero between launches
    const int *pos0;
    bf16 *cq, *ck, *cv;        // prompts: convolved queries and keys [tokens][kv_heads][dim], values [tokens][heads][vdim]
    uint8_t *rec;              // prompts: [tiles][heads] records
    float eps, out_mul, q_mul;
    int tokens, heads, kv_heads, dim, vdim, taps, k_at, v_at, g_at, a_at, ld, ld_ba, lda;
};

__device__ __forceinline__ int delta_channels(const DeltaArgs &a) { return 2 * a.kv_heads * a.dim + a.heads * a.vdim; }
// Input of channel c (column `col` of the projections) at token t of this call; t < 0: before it.
template <class AT>
__device__ __forceinline__ float delta_input(const DeltaArgs &a, int c, int col, int t, int pos0) {
    if (t >= 0) return to_f32(reinterpret_cast<const AT *>(a.p)[(size_t)t * a.ld + col]);
    const int pos = pos0 + t;
    return pos >= 0 ? a.ring[(size_t)(pos % delta_ring_rows(a.taps)) * delta_channels(a) + c] : 0.f;
}
// column of the projections that channel c comes from
__device__ __forceinline__ int delta_col(const DeltaArgs &a, int c) {
    const int qc = a.kv_heads * a.dim;
    return c < qc ? c : c < 2 * qc ? a.k_at + c - qc : a.v_at + c - 2 * qc;
}
// The inputs that the next call's convolutions reach back to, for channels first, first + step, ... < end
template <class AT>
__device__ __forceinline__ void delta_ring_store(const DeltaArgs &a, int first, int step, int end, int pos0) {
    const int C = delta_channels(a), R = delta_ring_rows(a.taps);
    for (int c = first; c < end; c += step) {
        const int col = delta_col(a, c);
        for (int t = max(0, a.tokens - a.taps + 1); t < a.tokens; t++)
            a.ring[(size_t)((pos0 + t) % R) * C + c] = to_f32(reinterpret_cast<const AT *>(a.p)[(size_t)t * a.ld + col]);
    }
}
// grid = ceil(channels / 256): the same as a launch of its own, behind everything that read the ring
template <class AT>
RNB_GLOBAL void __launch_bounds__(256)
delta_ring_kernel(const __grid_constant__ DeltaArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const int C = delta_channels(a), c = blockIdx.x * 256 + threadIdx.x;
    delta_ring_store<AT>(a, c, C, C, *a.pos0);
}

__host__ inline size_t delta_step_smem(int dim) { return sizeof(float) * (size_t)(DR_BLOCK * (2 * dim + 32) + 3 * DR_BLOCK + 8 * 64); }
// Block (h, jb) of heads x ceil(vdim / 32) = n_jb, 256 threads: lane = value column, warp w holds channels w, w + 8, ...
// (TI of them).  With act the block of a head that finishes last normalises and gates the head's outputs, and the ring is
// written (tokens <= 8).  Waits for the previous launch itself.
template <class AT, int TI>
__device__ __forceinline__ void delta_step_block(const DeltaArgs &a, int h, int jb, int n_jb, float *ds_smem) {
    const int dim = a.dim, vdim = a.vdim, j0 = jb * 32, rep = a.heads / a.kv_heads, hk = h / rep, C = delta_channels(a);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, j = j0 + lane, qc = a.kv_heads * dim;
    const bool live = j < vdim;
    float *sq = ds_smem, *sk = sq + DR_BLOCK * dim, *sv = sk + DR_BLOCK * dim, *sg = sv + DR_BLOCK * 32, *sb = sg + DR_BLOCK, *sqk = sb + DR_BLOCK, *red = sqk + DR_BLOCK;
    float *sp = a.state + (size_t)h * dim * vdim + j;
    if (vdim >= 32) {
        for (int ch = tid; ch < dim; ch += 256) asm volatile("prefetch.global.L2 [%0];" ::"l"(a.state + ((size_t)h * dim + ch) * vdim + j0));
    } else {
        prefetch_l2(a.state + (size_t)h * dim * vdim, (size_t)dim * vdim * 4, tid, 256);
    }
    for (int n = warp; n < a.taps; n += 8) {
        const float *w = a.conv + (size_t)n * C;
        prefetch_l2(w + hk * dim, (size_t)dim * 4, lane, 32);
        prefetch_l2(w + qc + hk * dim, (size_t)dim * 4, lane, 32);
        if (lane == 0) prefetch_l2(w + 2 * qc + h * vdim + j0, 4, 0, 1);
    }
    pdl_wait();
    float S[TI];
#pragma unroll
    for (int q = 0; q < TI; q++) {
        const int ch = warp + 8 * q;
        S[q] = live && ch < dim ? sp[(size_t)ch * vdim] : 0.f;
    }
    const int pos0 = *a.pos0;
    const float decay = -expf(a.a_log[h]), dt = a.dt[h];
    for (int t0 = 0; t0 < a.tokens; t0 += DR_BLOCK) {
        const int T = min(DR_BLOCK, a.tokens - t0);
        __syncthreads();
        // convolutions and silu: dim query channels, dim key channels, 32 value columns
        for (int i = tid; i < T * (2 * dim + 32); i += 256) {
            const int t = i / (2 * dim + 32), x = i % (2 * dim + 32);
            const int c = x < dim ? hk * dim + x : x < 2 * dim ? qc + hk * dim + x - dim : 2 * qc + h * vdim + j0 + x - 2 * dim;
            float y = 0.f;
            if (x < 2 * dim || j0 + x - 2 * dim < vdim) {
                const int col = delta_col(a, c);
#pragma unroll 4
                for (int n = 0; n < a.taps; n++) y = fmaf(a.conv[(size_t)n * C + c], delta_input<AT>(a, c, col, t0 + t - (a.taps - 1) + n, pos0), y);
                y = silu_f32(y);
            }
            if (x < dim) sq[t * dim + x] = y;
            else if (x < 2 * dim) sk[t * dim + x - dim] = y;
            else sv[t * 32 + x - 2 * dim] = y;
        }
        if (tid < T) {
            const float *ba = a.ba + (size_t)(t0 + tid) * a.ld_ba;
            sb[tid] = sigmoid_f32(ba[h]);
            sg[tid] = expm1f(decay * softplus_f32(ba[a.a_at + h] + dt));   // g - 1: over many tokens the rounding of a g near 1 adds up
        }
        __syncthreads();
        for (int t = warp; t < T; t += 8) {
            float qq = 0.f, kk = 0.f, qk = 0.f;
            for (int ch = lane; ch < dim; ch += 32) {
                const float x = sq[t * dim + ch], y = sk[t * dim + ch];
                qq = fmaf(x, x, qq), kk = fmaf(y, y, kk), qk = fmaf(x, y, qk);
            }
            const float b = a.q_mul / sqrtf(warp_sum(qq) + DR_UNIT_EPS), n = 1.0f / sqrtf(warp_sum(kk) + DR_UNIT_EPS);
            qk = warp_sum(qk);
            for (int ch = lane; ch < dim; ch += 32) sq[t * dim + ch] *= b, sk[t * dim + ch] *= n;
            if (lane == 0) sqk[t] = qk * b * n;
        }
        __syncthreads();
        for (int t = 0; t < T; t++) {
            const float g1 = sg[t];
            float kd = 0.f, qd = 0.f;
#pragma unroll
            for (int q = 0; q < TI; q++) {
                const int ch = warp + 8 * q;
                if (ch < dim) {
                    S[q] = fmaf(S[q], g1, S[q]);
                    kd = fmaf(sk[t * dim + ch], S[q], kd);
                    qd = fmaf(sq[t * dim + ch], S[q], qd);
                }
            }
            red[warp * 64 + lane] = kd;
            red[warp * 64 + 32 + lane] = qd;
            __syncthreads();
            kd = qd = 0.f;
#pragma unroll
            for (int i = 0; i < 8; i++) kd += red[i * 64 + lane], qd += red[i * 64 + 32 + lane];
            const float u = sb[t] * (sv[t * 32 + lane] - kd);
#pragma unroll
            for (int q = 0; q < TI; q++) {
                const int ch = warp + 8 * q;
                if (ch < dim) S[q] = fmaf(sk[t * dim + ch], u, S[q]);
            }
            if (warp == 0 && live) __stcg(a.o + ((size_t)(t0 + t) * a.heads + h) * vdim + j, fmaf(sqk[t], u, qd));
            __syncthreads();
        }
    }
#pragma unroll
    for (int q = 0; q < TI; q++) {
        const int ch = warp + 8 * q;
        if (live && ch < dim) sp[(size_t)ch * vdim] = S[q];
    }
    if (!a.act) return;
    // rows of this call's positions differ from those that other CTAs still read: the ring holds taps - 1 + 8
    if (h % rep == 0 && jb == 0) {
        delta_ring_store<AT>(a, hk * dim + tid, 256, (hk + 1) * dim, pos0);
        delta_ring_store<AT>(a, qc + hk * dim + tid, 256, qc + (hk + 1) * dim, pos0);
    }
    if (tid < 32) delta_ring_store<AT>(a, 2 * qc + h * vdim + j, 32, 2 * qc + h * vdim + min(j0 + 32, vdim), pos0);
    if (last_of_head(a.counters + h, n_jb))
        head_norm_gate_rows(a.o, reinterpret_cast<const float *>(a.p) + a.g_at, a.norm, a.act, a.tokens, a.heads, h, vdim, 0, a.ld, a.lda, a.eps, a.out_mul);
}

// grid = (heads, ceil(vdim / 32)), 256 threads
template <class AT, int TI>
RNB_GLOBAL void __launch_bounds__(256)
delta_step_kernel(const __grid_constant__ DeltaArgs a) {
    extern __shared__ __align__(16) float ds_smem[];
    pdl_launch_dependents();
    delta_step_block<AT, TI>(a, blockIdx.x, blockIdx.y, gridDim.y, ds_smem);
}

// ---- prompts on tensor cores ---------------------------------------------------------------------
// Record of a tile and head: T beta (bf16 hi, lo), P (hi, lo): 16 x 16 each, row t, column s; then f32: G_t0 a_t [16],
// G_t0 b_t [16], G_Tt a_t [16], G_T0 [1].
constexpr int DR_MAT = 16 * 16 * 2, DR_VEC = 4 * DR_MAT, DR_REC = DR_VEC + 4 * 64;
// tokens of a prepare CTA, and the pitch of its f32 matrices
constexpr int DP_TILES = 4, DP_TOKENS = 16 * DP_TILES, DP_PITCH = 20, DP_WORK = 16 * DP_PITCH + 32;
__host__ __device__ inline size_t delta_prepare_smem(int dim) {
    return (size_t)2 * DP_TOKENS * (dim + 8) * 2 + ((size_t)2 * DP_TILES * 16 * DP_PITCH + 2 * DP_TOKENS + 16 * DP_WORK) * 4;
}

// grid = (ceil(tokens / 64), kv_heads), 256 threads.  dim and vdim multiples of 8, dim of 16.
RNB_GLOBAL void __launch_bounds__(256, 2)
delta_prepare_kernel(const __grid_constant__ DeltaArgs a) {
    extern __shared__ __align__(16) uint8_t dp_smem[];
    pdl_launch_dependents();
    pdl_wait();
    const int dim = a.dim, rep = a.heads / a.kv_heads, hk = blockIdx.y, t0 = blockIdx.x * DP_TOKENS, nt = min(DP_TOKENS, a.tokens - t0), pos0 = *a.pos0;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, KE = dim + 8, qc = a.kv_heads * dim, C = delta_channels(a);
    bf16 *sx = reinterpret_cast<bf16 *>(dp_smem), *sy = sx + DP_TOKENS * KE;
    float *xy = reinterpret_cast<float *>(sy + DP_TOKENS * KE), *yy = xy + DP_TILES * 16 * DP_PITCH, *nrm = yy + DP_TILES * 16 * DP_PITCH, *work = nrm + 2 * DP_TOKENS;
    const bf16 *p = reinterpret_cast<const bf16 *>(a.p);
    // convolutions: 8 channels of 4 tokens at a time; rows past the end become zeros
    const int units = (2 * dim + rep * a.vdim) / 8;
    for (int i = tid; i < units * (DP_TOKENS / 4); i += 256) {
        const int u = i % units, ts = i / units * 4, x = u * 8;
        const int c = x < dim ? hk * dim + x : x < 2 * dim ? qc + hk * dim + x - dim : 2 * qc + hk * rep * a.vdim + x - 2 * dim;
        const int col = delta_col(a, c);
        float y[4][8] = {};
        for (int n = 0; n < a.taps; n++) {
            const float4 wa = *reinterpret_cast<const float4 *>(a.conv + (size_t)n * C + c), wb = *reinterpret_cast<const float4 *>(a.conv + (size_t)n * C + c + 4);
            const float w[8] = {wa.x, wa.y, wa.z, wa.w, wb.x, wb.y, wb.z, wb.w};
#pragma unroll
            for (int q = 0; q < 4; q++) {
                const int t = t0 + ts + q - (a.taps - 1) + n;
                if (ts + q >= nt) continue;
                float v[8];
                if (t >= 0) {
                    const uint4 b = *reinterpret_cast<const uint4 *>(p + (size_t)t * a.ld + col);
                    const uint32_t r[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
                    for (int e = 0; e < 4; e++) v[2 * e] = bf16_lo(r[e]), v[2 * e + 1] = bf16_hi(r[e]);
                } else {
#pragma unroll
                    for (int e = 0; e < 8; e++) v[e] = delta_input<bf16>(a, c + e, col + e, t, pos0);
                }
#pragma unroll
                for (int e = 0; e < 8; e++) y[q][e] = fmaf(w[e], v[e], y[q][e]);
            }
        }
#pragma unroll
        for (int q = 0; q < 4; q++) {
            const int t = ts + q;
            uint32_t r[4];
#pragma unroll
            for (int e = 0; e < 4; e++) r[e] = pg_pack_bf16(silu_fast(y[q][2 * e]), silu_fast(y[q][2 * e + 1]));
            const uint4 b = make_uint4(r[0], r[1], r[2], r[3]);
            if (x < 2 * dim) *reinterpret_cast<uint4 *>((x < dim ? sx + x : sy + x - dim) + t * KE) = b;
            if (t >= nt) continue;
            const size_t row = (size_t)(t0 + t);
            if (x < dim) *reinterpret_cast<uint4 *>(a.cq + (row * a.kv_heads + hk) * dim + x) = b;
            else if (x < 2 * dim) *reinterpret_cast<uint4 *>(a.ck + (row * a.kv_heads + hk) * dim + x - dim) = b;
            else *reinterpret_cast<uint4 *>(a.cv + (row * a.heads + hk * rep) * a.vdim + x - 2 * dim) = b;
        }
    }
    __syncthreads();
    // inverse norms, queries first, eight lanes per row
    for (int i = warp * 4 + (lane >> 3); i < 2 * DP_TOKENS; i += 32) {
        const bf16 *r = i < DP_TOKENS ? sx + i * KE : sy + (i - DP_TOKENS) * KE;
        float s = 0.f;
        for (int ch = (lane & 7) * 8; ch < dim; ch += 64) {
            const uint4 b = *reinterpret_cast<const uint4 *>(r + ch);
            const uint32_t v[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int e = 0; e < 4; e++) s = fmaf(bf16_lo(v[e]), bf16_lo(v[e]), s), s = fmaf(bf16_hi(v[e]), bf16_hi(v[e]), s);
        }
        for (int d = 1; d < 8; d <<= 1) s += __shfl_xor_sync(0xffffffffu, s, d);
        if ((lane & 7) == 0) nrm[i] = (i < DP_TOKENS ? a.q_mul : 1.0f) / sqrtf(s + DR_UNIT_EPS);
    }
    const int g = lane >> 2, tq = lane & 3, mi = lane >> 3, mr = lane & 7;
    {   // per tile x y^T (even warps) and y y^T (odd ones)
        const int tile = warp >> 1;
        float s[2][4] = {};
        const uint32_t pitch = (uint32_t)KE * 2, am = smem_u32((warp & 1 ? sy : sx) + tile * 16 * KE) + (uint32_t)((mi & 1) * 8 + mr) * pitch + (uint32_t)(mi >> 1) * 16u;
        const uint32_t bm = smem_u32(sy + tile * 16 * KE) + (uint32_t)((mi >> 1) * 8 + mr) * pitch + (uint32_t)(mi & 1) * 16u;
        for (int ks = 0; ks < dim / 16; ks++) {
            uint32_t fa[4], fb[4];
            lt_ldmatrix_x4(fa, am + (uint32_t)ks * 32u);
            lt_ldmatrix_x4(fb, bm + (uint32_t)ks * 32u);
            lt_mma(s[0], fa, fb[0], fb[1]);
            lt_mma(s[1], fa, fb[2], fb[3]);
        }
        float *out = (warp & 1 ? yy : xy) + tile * 16 * DP_PITCH;
#pragma unroll
        for (int n = 0; n < 2; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) out[(g + 8 * (e >> 1)) * DP_PITCH + n * 8 + 2 * tq + (e & 1)] = s[n][e];
    }
    __syncthreads();
    // half a warp per tile and head; lane s of it = column s of the matrices
    const int s = lane & 15, half = warp * 2 + (lane >> 4), tasks = min(DP_TILES, (nt + 15) / 16) * rep;
    float *M = work + half * DP_WORK, *lg = M + 16 * DP_PITCH, *bt = lg + 16;
    for (int base = 0; base < tasks; base += 16) {
        const int task = base + half;
        const bool on = task < tasks;
        const int tile = on ? task / rep : 0, h = hk * rep + (on ? task % rep : 0), tk = tile * 16, left = nt - tk;
        const float *nq = nrm + tk, *nk = nrm + DP_TOKENS + tk, *xt = xy + tile * 16 * DP_PITCH, *yt = yy + tile * 16 * DP_PITCH;
        const float *ba = a.ba + (size_t)(t0 + tk + min(s, left - 1)) * a.ld_ba;
        const float l = s < left ? -expf(a.a_log[h]) * softplus_f32(ba[a.a_at + h] + a.dt[h]) : 0.f, b = s < left ? sigmoid_f32(ba[h]) : 0.f;
        lg[s] = l;
        bt[s] = b;
        __syncwarp();
        uint8_t *rec = a.rec + ((size_t)(blockIdx.x * DP_TILES + tile) * a.heads + h) * DR_REC;
        bf16 *Thi = reinterpret_cast<bf16 *>(rec), *Tlo = Thi + 256, *Phi = Tlo + 256, *Plo = Phi + 256;
        float acc = 0.f, head = 0.f;   // logarithms of G_ts, and of G_s0
        const float ns = nk[s];
#pragma unroll
        for (int t = 0; t < 16; t++) {
            if (t <= s) head += lg[t];
            else acc += lg[t];
            const float e = t >= s ? expf(acc) * ns : 0.f;
            M[t * DP_PITCH + s] = t > s ? bt[t] * nk[t] * e * yt[t * DP_PITCH + s] : 0.f;
            if (on) lt_split_store(Phi + t * 16 + s, Plo + t * 16 + s, nq[t] * e * xt[t * DP_PITCH + s]);
        }
        if (on) {
            float *vec = reinterpret_cast<float *>(rec + DR_VEC);
            const float from0 = expf(head);
            vec[s] = from0 * ns;
            vec[16 + s] = from0 * nq[s];
            vec[32 + s] = expf(acc) * ns;
            if (s == 15) vec[48] = from0;
        }
        __syncwarp();
        // column s of (I + M)^-1 by forward substitution
        float x[16];
#pragma unroll
        for (int t = 0; t < 16; t++) {
            float v[4] = {t == s ? 1.f : 0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int q4 = 0; q4 < (t + 3) / 4; q4++) {
                const float4 m = *reinterpret_cast<const float4 *>(M + t * DP_PITCH + 4 * q4);
                const float mv[4] = {m.x, m.y, m.z, m.w};
#pragma unroll
                for (int e = 0; e < 4; e++)
                    if (4 * q4 + e < t) v[e] = fmaf(-mv[e], x[4 * q4 + e], v[e]);
            }
            x[t] = (v[0] + v[1]) + (v[2] + v[3]);
            if (on) lt_split_store(Thi + t * 16 + s, Tlo + t * 16 + s, x[t] * b);
        }
        __syncwarp();
    }
}

constexpr int DT_STAGES = 4;
__host__ __device__ constexpr int delta_tile_split(int DT) { return DT >= 4 ? 4 : 2; }   // warps that share the channels of 16 value columns
struct DeltaTileSmem {
    uint32_t kp, vp, y, v, mat, vec, stage, sums, bytes;
};
__host__ __device__ inline DeltaTileSmem delta_tile_smem(int DT, int CW) {
    DeltaTileSmem s;
    s.kp = (uint32_t)(16 * DT + 8) * 2;
    s.vp = (uint32_t)(16 * CW + 8) * 2;
    s.y = 16 * s.kp;                 // x at 0
    s.v = s.y + 16 * s.kp;
    s.mat = s.v + 16 * s.vp;         // four matrices, rows of 48 bytes
    s.vec = s.mat + 4 * 16 * 48;
    s.stage = s.vec + 256;
    s.sums = DT_STAGES * s.stage;    // partial products [2][CW][split][4][32 lanes] float4
    s.bytes = s.sums + (uint32_t)(2 * CW * delta_tile_split(DT) * 4 * 32 * 16);
    return s;
}
// grid = (heads, column blocks), blockDim = 32 * split * CW: 16 value columns per group of `split` warps, each of which holds
// S^T for its share of the channels.  The products with the state are summed over the group through shared memory.
// dim <= 16 DT a multiple of 16, vdim of 8.
template <int DT>
RNB_GLOBAL void __launch_bounds__(256)
delta_tile_kernel(const __grid_constant__ DeltaArgs a) {
    extern __shared__ __align__(128) uint8_t dt_smem[];
    pdl_launch_dependents();
    pdl_wait();
    constexpr int KS = delta_tile_split(DT), DW = DT / KS;   // channel blocks of 16 per warp
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nthr = blockDim.x, CW = nthr / (32 * KS), grp = warp / KS, part = warp % KS;
    const DeltaTileSmem L = delta_tile_smem(DT, CW);
    const uint32_t base = smem_u32(dt_smem);
    const int h = blockIdx.x, j0 = blockIdx.y * 16 * CW, hk = h / (a.heads / a.kv_heads), n_tiles = (a.tokens + 15) / 16, vdim = a.vdim;
    const size_t ldk = (size_t)a.kv_heads * a.dim, ldv = (size_t)a.heads * vdim;
    const bf16 *xp = a.cq + (size_t)hk * a.dim, *yp = a.ck + (size_t)hk * a.dim, *vp = a.cv + (size_t)h * vdim;
    auto cp16 = [&](uint32_t dst, const void *src, bool in) {
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(in ? 16u : 0u) : "memory");
    };
    auto load_tile = [&](int i) {
        if (i < n_tiles) {
            const uint32_t st = base + (uint32_t)(i % DT_STAGES) * L.stage;
            const int t0 = 16 * i;
            for (int x = tid; x < 16 * 2 * DT; x += nthr) {
                const int t = x / (2 * DT), q = x % (2 * DT);
                const bool in = t0 + t < a.tokens && q * 8 < a.dim;
                const size_t at = (size_t)min(t0 + t, a.tokens - 1) * ldk + min(q * 8, a.dim - 8);
                cp16(st + (uint32_t)t * L.kp + (uint32_t)q * 16u, xp + at, in);
                cp16(st + L.y + (uint32_t)t * L.kp + (uint32_t)q * 16u, yp + at, in);
            }
            for (int x = tid; x < 16 * 2 * CW; x += nthr) {
                const int t = x & 15, q = x >> 4, col = j0 + q * 8;
                cp16(st + L.v + (uint32_t)t * L.vp + (uint32_t)q * 16u, vp + (size_t)min(t0 + t, a.tokens - 1) * ldv + min(col, vdim - 8), t0 + t < a.tokens && col < vdim);
            }
            const uint8_t *rec = a.rec + ((size_t)i * a.heads + h) * DR_REC;
            for (int x = tid; x < DR_REC / 16; x += nthr)
                cp16(x < DR_VEC / 16 ? st + L.mat + (uint32_t)(x >> 1) * 48u + (uint32_t)(x & 1) * 16u : st + L.vec + (uint32_t)(x - DR_VEC / 16) * 16u, rec + x * 16, true);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    for (int i = 0; i < DT_STAGES - 1; i++) load_tile(i);
    {   // the ring for the next call's convolutions: every column block takes its share of the head's channels
        const int rep = a.heads / a.kv_heads, qc = a.kv_heads * a.dim, pos0 = *a.pos0, step = nthr * gridDim.y, first = blockIdx.y * nthr + tid;
        if (h % rep == 0) {
            delta_ring_store<bf16>(a, hk * a.dim + first, step, (hk + 1) * a.dim, pos0);
            delta_ring_store<bf16>(a, qc + hk * a.dim + first, step, qc + (hk + 1) * a.dim, pos0);
        }
        delta_ring_store<bf16>(a, 2 * qc + h * vdim + first, step, 2 * qc + (h + 1) * vdim, pos0);
    }
    const int g = lane >> 2, tq = lane & 3, mi = lane >> 3, mr = lane & 7, jw = j0 + grp * 16, c0 = part * DW * 16;
    float S[2 * DW][4];
    auto state_io = [&](bool store) {
#pragma unroll
        for (int n = 0; n < 2 * DW; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int ch = c0 + n * 8 + 2 * tq + (e & 1), j = jw + g + 8 * (e >> 1);
                const bool in = j < vdim && ch < a.dim;
                float *p = a.state + ((size_t)h * a.dim + ch) * vdim + j;
                if (store) {
                    if (in) *p = S[n][e];
                } else {
                    S[n][e] = in ? *p : 0.f;
                }
            }
    };
    state_io(false);
    const uint32_t b_plain = (uint32_t)((mi >> 1) * 8 + mr) * L.kp + (uint32_t)(mi & 1) * 16u + (uint32_t)c0 * 2u;        // rows (n), k contiguous
    const uint32_t b_trans = (uint32_t)((mi & 1) * 8 + mr) * L.kp + (uint32_t)(mi >> 1) * 16u + (uint32_t)c0 * 2u;        // rows (k), n contiguous
    const uint32_t b_mat = (uint32_t)((mi >> 1) * 8 + mr) * 48u + (uint32_t)(mi & 1) * 16u;
    float4 *sums = reinterpret_cast<float4 *>(dt_smem + L.sums) + (size_t)grp * KS * 128;
    for (int it = 0; it < n_tiles; it++) {
        asm volatile("cp.async.wait_group %0;" ::"n"(DT_STAGES - 2) : "memory");
        __syncthreads();   // the tile is in, and every warp is through with the one whose stage is loaded next
        load_tile(it + DT_STAGES - 1);
        const uint32_t st = base + (uint32_t)(it % DT_STAGES) * L.stage;
        const uint8_t *raw = dt_smem + (size_t)(it % DT_STAGES) * L.stage;
        const float *vec = reinterpret_cast<const float *>(raw + L.vec);
        // this warp's part of (S0^T y, S0^T x): state hi + lo, exact bf16 rows
        float X[4][4] = {}, Y[4][4] = {};
#pragma unroll
        for (int ks = 0; ks < DW; ks++) {
            uint32_t sh[4], sl[4], by[4], bx[4];
            lt_split(S[2 * ks][0], S[2 * ks][1], sh[0], sl[0]);
            lt_split(S[2 * ks][2], S[2 * ks][3], sh[1], sl[1]);
            lt_split(S[2 * ks + 1][0], S[2 * ks + 1][1], sh[2], sl[2]);
            lt_split(S[2 * ks + 1][2], S[2 * ks + 1][3], sh[3], sl[3]);
            lt_ldmatrix_x4(by, st + L.y + b_plain + (uint32_t)ks * 32u);
            lt_ldmatrix_x4(bx, st + b_plain + (uint32_t)ks * 32u);
            lt_mma(X[0], sh, by[0], by[1]);
            lt_mma(X[1], sh, by[2], by[3]);
            lt_mma(X[2], sl, by[0], by[1]);
            lt_mma(X[3], sl, by[2], by[3]);
            lt_mma(Y[0], sh, bx[0], bx[1]);
            lt_mma(Y[1], sh, bx[2], bx[3]);
            lt_mma(Y[2], sl, bx[0], bx[1]);
            lt_mma(Y[3], sl, bx[2], bx[3]);
        }
        float4 *mine = sums + (size_t)(it & 1) * CW * KS * 128, *put = mine + part * 128 + lane;
#pragma unroll
        for (int n = 0; n < 2; n++) {
            put[n * 32] = make_float4(X[n][0] + X[n + 2][0], X[n][1] + X[n + 2][1], X[n][2] + X[n + 2][2], X[n][3] + X[n + 2][3]);
            put[(n + 2) * 32] = make_float4(Y[n][0] + Y[n + 2][0], Y[n][1] + Y[n + 2][1], Y[n][2] + Y[n + 2][2], Y[n][3] + Y[n + 2][3]);
        }
        asm volatile("bar.sync %0, %1;" ::"r"(1 + grp), "n"(32 * KS) : "memory");
        auto total = [&](int n, float (&o)[4]) {
            o[0] = o[1] = o[2] = o[3] = 0.f;
#pragma unroll
            for (int k = 0; k < KS; k++) {
                const float4 v = mine[k * 128 + n * 32 + lane];
                o[0] += v.x, o[1] += v.y, o[2] += v.z, o[3] += v.w;
            }
        };
        // V - G_t0 a_t S0^T y
        const bf16 *sv = reinterpret_cast<const bf16 *>(raw + L.v);
        const int VE = (int)(L.vp / 2);
        float R[2][4];
#pragma unroll
        for (int n = 0; n < 2; n++) {
            float x[4];
            total(n, x);
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int t = n * 8 + 2 * tq + (e & 1);
                R[n][e] = fmaf(-vec[t], x[e], to_f32(sv[t * VE + grp * 16 + g + 8 * (e >> 1)]));
            }
        }
        auto split_tile = [&](const float (&m)[2][4], uint32_t (&hi)[4], uint32_t (&lo)[4]) {
            lt_split(m[0][0], m[0][1], hi[0], lo[0]);
            lt_split(m[0][2], m[0][3], hi[1], lo[1]);
            lt_split(m[1][0], m[1][1], hi[2], lo[2]);
            lt_split(m[1][2], m[1][3], hi[3], lo[3]);
        };
        uint32_t hi[4], lo[4], bh[4], bl[4];
        split_tile(R, hi, lo);
        lt_ldmatrix_x4(bh, st + L.mat + b_mat);
        lt_ldmatrix_x4(bl, st + L.mat + 16 * 48 + b_mat);
        float U[2][4] = {}, U2[2][4] = {}, W[2][4];
        lt_mma(U[0], hi, bh[0], bh[1]);
        lt_mma(U[1], hi, bh[2], bh[3]);
        lt_mma(U2[0], lo, bh[0], bh[1]);
        lt_mma(U2[1], lo, bh[2], bh[3]);
        lt_mma(U2[0], hi, bl[0], bl[1]);
        lt_mma(U2[1], hi, bl[2], bl[3]);
#pragma unroll
        for (int n = 0; n < 2; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                U[n][e] += U2[n][e];
                W[n][e] = U[n][e] * vec[32 + n * 8 + 2 * tq + (e & 1)];
            }
        // the state moves on first: the next tile waits for it
        uint32_t wh[4], wl[4];
        split_tile(W, wh, wl);
        const float decay = vec[48];
#pragma unroll
        for (int np = 0; np < DW; np++) {
            uint32_t kb[4];
            lt_ldmatrix_x4_trans(kb, st + L.y + b_trans + (uint32_t)np * 32u);
#pragma unroll
            for (int e = 0; e < 4; e++) S[2 * np][e] *= decay, S[2 * np + 1][e] *= decay;
            lt_mma(S[2 * np], wh, kb[0], kb[1]);
            lt_mma(S[2 * np + 1], wh, kb[2], kb[3]);
            lt_mma(S[2 * np], wl, kb[0], kb[1]);
            lt_mma(S[2 * np + 1], wl, kb[2], kb[3]);
        }
        // outputs: two warps of the group take eight tokens each
        if (part < 2) {
            float o[4];
            total(2 + part, o);
#pragma unroll
            for (int e = 0; e < 4; e++) o[e] *= vec[16 + part * 8 + 2 * tq + (e & 1)];
            split_tile(U, hi, lo);
            lt_ldmatrix_x4(bh, st + L.mat + 2 * 16 * 48 + b_mat);
            lt_ldmatrix_x4(bl, st + L.mat + 3 * 16 * 48 + b_mat);
            const uint32_t h0 = part ? bh[2] : bh[0], h1 = part ? bh[3] : bh[1], l0 = part ? bl[2] : bl[0], l1 = part ? bl[3] : bl[1];
            lt_mma(o, hi, h0, h1);
            lt_mma(o, lo, h0, h1);
            lt_mma(o, hi, l0, l1);
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int t = 16 * it + part * 8 + 2 * tq + (e & 1), j = jw + g + 8 * (e >> 1);
                if (t < a.tokens && j < vdim) a.o[((size_t)t * a.heads + h) * vdim + j] = o[e];
            }
        }
    }
    state_io(true);
}

}  // namespace rnb
