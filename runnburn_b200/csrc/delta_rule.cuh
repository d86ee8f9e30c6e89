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
//   R = V - (G_t0 a_t y_t) S0,   U = N R with N = (I + M)^-1 beta,   M_ts = beta_t G_ts a_t a_s (y_t . y_s) for s < t
//   o_t = b_t G_t0 x_t S0 + (P U)_t with P_ts = b_t G_ts a_s (x_t . y_s) for s <= t,   S = G_T0 S0 + sum_s y_s (G_Ts a_s u_s)^T
// so that the matrices (G_Ts a_s) N and P N of a tile do not depend on the state and are made ahead of time.
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
    // prompts, as shared memory wants a tile (16 tokens): convolved queries and keys [tiles][kv_heads][2][16][ld_qk], values
    // [tiles][heads][col_blocks][16][ld_val] (16 cw columns per block), records [tiles][heads]
    bf16 *cqk, *cv;
    uint8_t *rec;
    int *err;                  // prompts: device error flag
    float eps, out_mul, q_mul;
    int tokens, heads, kv_heads, dim, vdim, taps, k_at, v_at, g_at, a_at, ld, ld_ba, lda, ld_qk, ld_val, col_blocks, cw;
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
    if (a.norm) prefetch_l2(a.norm, (size_t)vdim * 4, tid, 256);
    pdl_wait();
    float S[TI];
#pragma unroll
    for (int q = 0; q < TI; q++) {
        const int ch = warp + 8 * q;
        S[q] = live && ch < dim ? sp[(size_t)ch * vdim] : 0.f;
    }
    const int pos0 = *a.pos0, R = delta_ring_rows(a.taps), slot0 = (pos0 + R - (a.taps - 1)) % R;   // where position pos0 - (taps - 1) lies
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
                const AT *in = reinterpret_cast<const AT *>(a.p) + delta_col(a, c);
                const int before = max(0, a.taps - 1 - (t0 + t));   // taps that reach back past this call
                int slot = slot0 + t0 + t;
                if (slot >= R) slot -= R;
#pragma unroll 4
                for (int n = 0; n < a.taps; n++) {
                    const float w = a.conv[(size_t)n * C + c];
                    float v;
                    if (n >= before) v = to_f32(in[(size_t)(t0 + t - (a.taps - 1) + n) * a.ld]);
                    else v = pos0 + t0 + t - (a.taps - 1) + n >= 0 ? a.ring[(size_t)slot * C + c] : 0.f;
                    if (++slot == R) slot = 0;
                    y = fmaf(w, v, y);
                }
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
// Record of a tile and head: (G_Tt a_t) N (bf16 hi, lo), P N (hi, lo): 16 x 16 each, row t, column s; then f32:
// G_t0 a_t [16], G_t0 b_t [16], G_T0 [1].
constexpr int DR_ROW = 48, DR_MAT = 16 * DR_ROW, DR_VEC = 4 * DR_MAT, DR_REC = DR_VEC + 4 * 64;   // rows of 48 bytes: the form shared memory wants
// tokens of a prepare CTA, and the pitch of its f32 matrices
constexpr int DP_TILES = 4, DP_TOKENS = 16 * DP_TILES, DP_PITCH = 20, DP_WORK = 2 * 16 * DP_PITCH + 16;
__host__ __device__ inline size_t delta_prepare_smem(int dim) {
    return (size_t)2 * DP_TOKENS * (dim + 8) * 2 + ((size_t)2 * DP_TILES * 16 * DP_PITCH + 2 * DP_TOKENS + 16 * DP_WORK) * 4;
}

// Convolution and silu of 8 channels (column `col` of the projections, taps from channel c on) at the 16 tokens from t on:
// put(i, eight bf16) for each of them, zeros from token `end` on.  TAPS: their number, 0 for any.
template <int TAPS, class Put>
__device__ __forceinline__ void delta_convolve16(const DeltaArgs &a, int c, int col, int t, int end, int pos0, Put put) {
    const int taps = TAPS ? TAPS : a.taps, C = delta_channels(a);
    const bf16 *p = reinterpret_cast<const bf16 *>(a.p) + col;
    auto load = [&](int at) { return *reinterpret_cast<const uint4 *>(p + (size_t)min(at, a.tokens - 1) * a.ld); };
    auto unpack = [&](uint4 b, float (&v)[8]) {
        const uint32_t r[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
        for (int e = 0; e < 4; e++) v[2 * e] = bf16_lo(r[e]), v[2 * e + 1] = bf16_hi(r[e]);
    };
    auto row = [&](int at, float (&v)[8]) {
        if (at >= 0) unpack(load(at), v);
        else
            for (int e = 0; e < 8; e++) v[e] = delta_input<bf16>(a, c + e, col + e, at, pos0);
    };
    auto weights = [&](int n, float (&w)[8]) {
        const float4 x = *reinterpret_cast<const float4 *>(a.conv + (size_t)n * C + c), y = *reinterpret_cast<const float4 *>(a.conv + (size_t)n * C + c + 4);
        w[0] = x.x, w[1] = x.y, w[2] = x.z, w[3] = x.w, w[4] = y.x, w[5] = y.y, w[6] = y.z, w[7] = y.w;
    };
    auto finish = [&](int i, const float (&y)[8]) {
        uint32_t r[4] = {0u, 0u, 0u, 0u};
        if (t + i < end) {
#pragma unroll
            for (int e = 0; e < 4; e++) r[e] = pg_pack_bf16(silu_fast(y[2 * e]), silu_fast(y[2 * e + 1]));
        }
        put(i, make_uint4(r[0], r[1], r[2], r[3]));
    };
    if (TAPS) {
        // groups of N tokens: their rows are asked for a group ahead, and the last rows form a ring whose places are known
        constexpr int N = TAPS ? TAPS : 1;
        float w[N][8], x[N][8];
        uint4 next[N];
#pragma unroll
        for (int n = 0; n < N; n++) next[n] = load(t + n);
#pragma unroll
        for (int n = 0; n < N; n++) weights(n, w[n]);
#pragma unroll
        for (int n = 0; n < N - 1; n++) row(t - (N - 1) + n, x[n]);
#pragma unroll 1
        for (int i0 = 0; i0 < 16; i0 += N) {
            uint4 now[N];
#pragma unroll
            for (int n = 0; n < N; n++) now[n] = next[n];
            if (i0 + N < 16)
#pragma unroll
                for (int n = 0; n < N; n++) next[n] = load(t + i0 + N + n);
#pragma unroll
            for (int i = 0; i < N; i++) {
                if (i0 + i >= 16) break;
                unpack(now[i], x[(i + N - 1) % N]);
                float y[8] = {};
#pragma unroll
                for (int n = 0; n < N; n++)
#pragma unroll
                    for (int e = 0; e < 8; e++) y[e] = fmaf(w[n][e], x[(i + n) % N][e], y[e]);
                finish(i0 + i, y);
            }
        }
    } else {
        for (int i = 0; i < 16; i++) {
            float y[8] = {};
            for (int n = 0; n < taps; n++) {
                float w[8], x[8];
                weights(n, w);
                row(t + i - (taps - 1) + n, x);
#pragma unroll
                for (int e = 0; e < 8; e++) y[e] = fmaf(w[e], x[e], y[e]);
            }
            finish(i, y);
        }
    }
}

// grid = (ceil(tokens / 64), kv_heads), 256 threads.  dim and vdim multiples of 8, dim of 16.
template <int TAPS>
RNB_GLOBAL void __launch_bounds__(256, 2)
delta_prepare_kernel(const __grid_constant__ DeltaArgs a) {
    extern __shared__ __align__(16) uint8_t dp_smem[];
    pdl_launch_dependents();
    pdl_wait();
    const int dim = a.dim, rep = a.heads / a.kv_heads, hk = blockIdx.y, t0 = blockIdx.x * DP_TOKENS, nt = min(DP_TOKENS, a.tokens - t0), pos0 = *a.pos0;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, KE = dim + 8, qc = a.kv_heads * dim;
    bf16 *sx = reinterpret_cast<bf16 *>(dp_smem), *sy = sx + DP_TOKENS * KE;
    float *xy = reinterpret_cast<float *>(sy + DP_TOKENS * KE), *yy = xy + DP_TILES * 16 * DP_PITCH, *nrm = yy + DP_TILES * 16 * DP_PITCH, *work = nrm + 2 * DP_TOKENS;
    // convolutions: 8 channels of a tile at a time; rows past the end become zeros
    const int units = (2 * dim + rep * a.vdim) / 8;
    for (int i = tid; i < units * DP_TILES; i += 256) {
        const int u = i % units, ts = i / units * 16, x = u * 8;
        if (ts >= nt) {   // no such tile: only the rows that the products below read
            if (x < 2 * dim)
                for (int k = 0; k < 16; k++) *reinterpret_cast<uint4 *>((x < dim ? sx + x : sy + x - dim) + (ts + k) * KE) = make_uint4(0u, 0u, 0u, 0u);
            continue;
        }
        const int c = x < dim ? hk * dim + x : x < 2 * dim ? qc + hk * dim + x - dim : 2 * qc + hk * rep * a.vdim + x - 2 * dim;
        const size_t tile = (size_t)blockIdx.x * DP_TILES + (i / units);
        bf16 *near = nullptr, *far;
        int ld = a.ld_qk;
        if (x < 2 * dim) {
            const int key = x >= dim, ch = key ? x - dim : x;
            near = (key ? sy : sx) + ts * KE + ch;
            far = a.cqk + ((tile * a.kv_heads + hk) * 2 + key) * 16 * ld + ch;
        } else {
            const int j = (x - 2 * dim) % a.vdim, h = hk * rep + (x - 2 * dim) / a.vdim, w = 16 * a.cw;
            ld = a.ld_val;
            far = a.cv + ((tile * a.heads + h) * a.col_blocks + j / w) * 16 * ld + j % w;
        }
        delta_convolve16<TAPS>(a, c, delta_col(a, c), t0 + ts, a.tokens, pos0, [&](int k, uint4 b) {
            if (near) *reinterpret_cast<uint4 *>(near + k * KE) = b;
            *reinterpret_cast<uint4 *>(far + k * ld) = b;
        });
    }
    if (dim + 8 < a.ld_qk) {   // channels that the tile kernel has beyond dim
        const int pad = (a.ld_qk - 8 - dim) / 8, rows = (nt + 15) / 16 * 32;
        for (int i = tid; i < rows * pad; i += 256)
            *reinterpret_cast<uint4 *>(a.cqk + (((size_t)(blockIdx.x * DP_TILES + i / pad / 32) * a.kv_heads + hk) * 32 + i / pad % 32) * a.ld_qk + dim + i % pad * 8) = make_uint4(0u, 0u, 0u, 0u);
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
    float *M = work + half * DP_WORK, *P = M + 16 * DP_PITCH, *lg = P + 16 * DP_PITCH;
    for (int base = 0; base < tasks; base += 16) {
        const int task = base + half;
        const bool on = task < tasks;
        const int tile = on ? task / rep : 0, h = hk * rep + (on ? task % rep : 0), tk = tile * 16, left = nt - tk;
        const float *nq = nrm + tk, *nk = nrm + DP_TOKENS + tk, *xt = xy + tile * 16 * DP_PITCH, *yt = yy + tile * 16 * DP_PITCH;
        const float *ba = a.ba + (size_t)(t0 + tk + min(s, left - 1)) * a.ld_ba;
        const float b = s < left ? sigmoid_f32(ba[h]) : 0.f;
        lg[s] = s < left ? -expf(a.a_log[h]) * softplus_f32(ba[a.a_at + h] + a.dt[h]) : 0.f;
        __syncwarp();
        uint8_t *rec = a.rec + ((size_t)(blockIdx.x * DP_TILES + tile) * a.heads + h) * DR_REC;
        constexpr int RE = DR_ROW / 2, ME = DR_MAT / 2;
        bf16 *Whi = reinterpret_cast<bf16 *>(rec), *Wlo = Whi + ME, *Qhi = Wlo + ME, *Qlo = Qhi + ME;
        float acc = 0.f, head = 0.f;   // logarithms of G_ts, and of G_s0
        const float ns = nk[s];
#pragma unroll
        for (int t = 0; t < 16; t++) {
            if (t <= s) head += lg[t];
            else acc += lg[t];
            const float e = t >= s ? expf(acc) * ns : 0.f;
            const float bt = __shfl_sync(0xffffffffu, b, t, 16);
            M[t * DP_PITCH + s] = t > s ? bt * nk[t] * e * yt[t * DP_PITCH + s] : 0.f;
            P[t * DP_PITCH + s] = nq[t] * e * xt[t * DP_PITCH + s];
        }
        const float from0 = expf(head), to_end = expf(acc) * ns;
        if (on) {
            float *vec = reinterpret_cast<float *>(rec + DR_VEC);
            vec[s] = from0 * ns;
            vec[16 + s] = from0 * nq[s];
            if (s == 15) vec[32] = from0;
        }
        __syncwarp();
        // column s of N by forward substitution
        float x[16];
        auto dot = [&](const float *row, int n, float first) {   // first + the first n elements of a row times x
            float v[4] = {first, 0.f, 0.f, 0.f};
#pragma unroll
            for (int q4 = 0; q4 < 4; q4++) {
                if (4 * q4 >= n) break;
                const float4 m = *reinterpret_cast<const float4 *>(row + 4 * q4);
                const float mv[4] = {m.x, m.y, m.z, m.w};
#pragma unroll
                for (int e = 0; e < 4; e++)
                    if (4 * q4 + e < n) v[e] = fmaf(mv[e], x[4 * q4 + e], v[e]);
            }
            return (v[0] + v[1]) + (v[2] + v[3]);
        };
#pragma unroll
        for (int t = 0; t < 16; t++) x[t] = (t == s ? b : 0.f) - dot(M + t * DP_PITCH, t, 0.f);
#pragma unroll
        for (int t = 0; t < 16; t++) {
            const float q = dot(P + t * DP_PITCH, t + 1, 0.f), w = __shfl_sync(0xffffffffu, to_end, t, 16) * x[t];
            if (!on) continue;
            lt_split_store(Whi + t * RE + s, Wlo + t * RE + s, w);
            lt_split_store(Qhi + t * RE + s, Qlo + t * RE + s, q);
        }
        __syncwarp();
    }
}

constexpr int DT_STAGES = 4, DT_SPLIT = 2;   // DT_SPLIT: warps that share the channels of 16 value columns (and the two halves of a tile's tokens)
struct DeltaTileSmem {
    uint32_t kp, vp, y, v, mat, vec, stage, sums, bytes;
};
__host__ __device__ inline DeltaTileSmem delta_tile_smem(int DT, int CW) {
    DeltaTileSmem s;
    s.kp = (uint32_t)(16 * DT + 8) * 2;
    s.vp = (uint32_t)(16 * CW + 8) * 2;
    s.y = 16 * s.kp;                 // x at 0
    s.v = s.y + 16 * s.kp;
    s.mat = s.v + 16 * s.vp;         // four matrices, rows of 48 bytes, then the record's vectors
    s.vec = s.mat + DR_VEC;
    s.stage = s.mat + DR_REC;
    s.sums = DT_STAGES * s.stage;    // partial products [2][CW][split][4][32 lanes] float4
    s.bytes = s.sums + (uint32_t)(2 * CW * DT_SPLIT * 4 * 32 * 16);
    return s;
}
// grid = (heads, column blocks), blockDim = 32 * (DT_SPLIT * cw + 1): 16 value columns per group of DT_SPLIT warps, each of which
// holds S^T for its share of the channels; the last warp has a tile's queries and keys, values and record copied into a ring of stages
// (three bulk copies).  The products with the state are summed over the group through shared memory; each warp finishes eight of a
// tile's tokens.
// Waits are bounded; one that gives up sets the error flag, and every copy that was started is waited for before the CTA ends.
// dim <= 16 DT a multiple of 16, vdim of 8.
template <int DT>
RNB_GLOBAL void __launch_bounds__(160)
delta_tile_kernel(const __grid_constant__ DeltaArgs a) {
    extern __shared__ __align__(128) uint8_t dt_smem[];
    __shared__ __align__(8) uint64_t full[DT_STAGES], empty[DT_STAGES];
    __shared__ int s_failed;
    pdl_launch_dependents();
    constexpr int KS = DT_SPLIT, DW = DT / KS;   // channel blocks of 16 per warp
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, CW = a.cw, grp = warp / KS, part = warp % KS;
    const DeltaTileSmem L = delta_tile_smem(DT, CW);
    const uint32_t base = smem_u32(dt_smem);
    const int h = blockIdx.x, j0 = blockIdx.y * 16 * CW, hk = h / (a.heads / a.kv_heads), n_tiles = (a.tokens + 15) / 16, vdim = a.vdim;
    const size_t ldv = (size_t)a.heads * vdim;
    if (tid == 0) {
        for (int i = 0; i < DT_STAGES; i++) {
            mbar_init(&full[i], 1);
            mbar_init(&empty[i], (uint32_t)(KS * CW));
        }
        mbar_fence_init();
        s_failed = 0;
    }
    __syncthreads();
    pdl_wait();
    if (warp == KS * CW) {
        int issued = 0;
        bool ok = true;
        if (lane == 0) {
            const uint32_t qk = 32 * L.kp, val = 16 * L.vp;
            for (int i = 0; i < n_tiles; i++) {
                const int sl = i % DT_STAGES;
                ok = mbar_wait_bounded(&empty[sl], (uint32_t)(((i / DT_STAGES) & 1) ^ 1));
                if (!ok) break;
                uint8_t *st = dt_smem + (size_t)sl * L.stage;
                mbar_arrive_expect_tx(&full[sl], qk + val + DR_REC);
                bulk_g2s(st, a.cqk + ((size_t)i * a.kv_heads + hk) * 32 * a.ld_qk, qk, &full[sl]);
                bulk_g2s(st + L.v, a.cv + (((size_t)i * a.heads + h) * a.col_blocks + blockIdx.y) * 16 * a.ld_val, val, &full[sl]);
                bulk_g2s(st + L.mat, a.rec + ((size_t)i * a.heads + h) * DR_REC, DR_REC, &full[sl]);
                issued = i + 1;
            }
        }
        if (!ok && lane == 0) atomicExch(&s_failed, 1);
        // a CTA ends after its copies
        for (int i = max(0, issued - DT_STAGES); i < issued; i++) mbar_wait_bounded(&full[i % DT_STAGES], (uint32_t)((i / DT_STAGES) & 1));
    } else {
        {   // the ring for the next call's convolutions: every column block takes its share of the head's channels
            const int rep = a.heads / a.kv_heads, qc = a.kv_heads * a.dim, pos0 = *a.pos0, step = 32 * KS * CW * gridDim.y, first = blockIdx.y * 32 * KS * CW + tid;
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
        const uint32_t b_mat = L.mat + (uint32_t)((mi >> 1) * 8 + mr) * DR_ROW + (uint32_t)(mi & 1) * 16u;
        const uint32_t b_out = L.mat + (uint32_t)(2 + (mi >> 1)) * DR_MAT + (uint32_t)(part * 8 + mr) * DR_ROW + (uint32_t)(mi & 1) * 16u;   // hi, lo of eight rows
        const uint32_t b_val = L.v + (uint32_t)((mi >> 1) * 8 + mr) * L.vp + (uint32_t)(grp * 32 + (mi & 1) * 16);
        float4 *sums = reinterpret_cast<float4 *>(dt_smem + L.sums) + (size_t)grp * KS * 128 + lane;
        float *to = a.o + (size_t)(part * 8 + 2 * tq) * ldv + (size_t)h * vdim + jw + g;
        const bool col0 = jw + g < vdim, col1 = jw + g + 8 < vdim;
        bool ok = true;
        for (int it = 0; it < n_tiles; it++, to += 16 * ldv) {
            const int sl = it % DT_STAGES;
            if (ok) ok = mbar_wait_bounded(&full[sl], (uint32_t)((it / DT_STAGES) & 1));
            ok = __all_sync(0xffffffffu, ok);
            const uint32_t st = base + (uint32_t)sl * L.stage;
            const float *vec = reinterpret_cast<const float *>(dt_smem + (size_t)sl * L.stage + L.vec);
            // this warp's part of (S0^T y, S0^T x): state hi + lo, exact bf16 rows
            float X[4][4], Y[4][4];
#pragma unroll
            for (int ks = 0; ks < DW; ks++) {
                uint32_t sh[4], s2[4], by[4], bx[4];
                lt_ldmatrix_x4(by, st + L.y + b_plain + (uint32_t)ks * 32u);
                lt_ldmatrix_x4(bx, st + b_plain + (uint32_t)ks * 32u);
                lt_split(S[2 * ks][0], S[2 * ks][1], sh[0], s2[0]);
                lt_split(S[2 * ks][2], S[2 * ks][3], sh[1], s2[1]);
                lt_split(S[2 * ks + 1][0], S[2 * ks + 1][1], sh[2], s2[2]);
                lt_split(S[2 * ks + 1][2], S[2 * ks + 1][3], sh[3], s2[3]);
                if (ks == 0) {
                    lt_mma_zero(X[0], sh, by[0], by[1]);
                    lt_mma_zero(X[1], sh, by[2], by[3]);
                    lt_mma_zero(X[2], s2, by[0], by[1]);
                    lt_mma_zero(X[3], s2, by[2], by[3]);
                    lt_mma_zero(Y[0], sh, bx[0], bx[1]);
                    lt_mma_zero(Y[1], sh, bx[2], bx[3]);
                    lt_mma_zero(Y[2], s2, bx[0], bx[1]);
                    lt_mma_zero(Y[3], s2, bx[2], bx[3]);
                } else {
                    lt_mma(X[0], sh, by[0], by[1]);
                    lt_mma(X[1], sh, by[2], by[3]);
                    lt_mma(X[2], s2, by[0], by[1]);
                    lt_mma(X[3], s2, by[2], by[3]);
                    lt_mma(Y[0], sh, bx[0], bx[1]);
                    lt_mma(Y[1], sh, bx[2], bx[3]);
                    lt_mma(Y[2], s2, bx[0], bx[1]);
                    lt_mma(Y[3], s2, bx[2], bx[3]);
                }
            }
            float4 *box = sums + (size_t)(it & 1) * CW * KS * 128;
#pragma unroll
            for (int n = 0; n < 2; n++) {
                box[part * 128 + n * 32] = make_float4(X[n][0] + X[n + 2][0], X[n][1] + X[n + 2][1], X[n][2] + X[n + 2][2], X[n][3] + X[n + 2][3]);
                box[part * 128 + 64 + n * 32] = make_float4(Y[n][0] + Y[n + 2][0], Y[n][1] + Y[n + 2][1], Y[n][2] + Y[n + 2][2], Y[n][3] + Y[n + 2][3]);
            }
            uint32_t v4[4], bh[4], bl[4];
            lt_ldmatrix_x4_trans(v4, st + b_val);
            lt_ldmatrix_x4(bh, st + b_mat);
            lt_ldmatrix_x4(bl, st + b_mat + DR_MAT);
            asm volatile("bar.sync %0, %1;" ::"r"(1 + grp), "n"(32 * KS) : "memory");
            auto total = [&](int n) {
                float4 q = box[n * 32];
#pragma unroll
                for (int k = 1; k < KS; k++) {
                    const float4 v = box[k * 128 + n * 32];
                    q.x += v.x, q.y += v.y, q.z += v.z, q.w += v.w;
                }
                return q;
            };
            // R^T = V^T - G_t0 a_t S0^T y
            float R[2][4];
#pragma unroll
            for (int n = 0; n < 2; n++) {
                const float4 q = total(n);
                const float2 f = *reinterpret_cast<const float2 *>(vec + n * 8 + 2 * tq);
                R[n][0] = fmaf(-f.x, q.x, bf16_lo(v4[2 * n]));
                R[n][1] = fmaf(-f.y, q.y, bf16_hi(v4[2 * n]));
                R[n][2] = fmaf(-f.x, q.z, bf16_lo(v4[2 * n + 1]));
                R[n][3] = fmaf(-f.y, q.w, bf16_hi(v4[2 * n + 1]));
            }
            auto split_tile = [&](const float (&m)[2][4], uint32_t (&hi)[4], uint32_t (&lo)[4]) {
                lt_split(m[0][0], m[0][1], hi[0], lo[0]);
                lt_split(m[0][2], m[0][3], hi[1], lo[1]);
                lt_split(m[1][0], m[1][1], hi[2], lo[2]);
                lt_split(m[1][2], m[1][3], hi[3], lo[3]);
            };
            uint32_t hi[4], lo[4];
            split_tile(R, hi, lo);
            // products that add to the same accumulators lie a few issues apart; the rest of the work fills in
            float W[2][4], W2[2][4];
            lt_mma_zero(W2[0], lo, bh[0], bh[1]);
            lt_mma_zero(W2[1], lo, bh[2], bh[3]);
            lt_mma_zero(W[0], hi, bh[0], bh[1]);
            lt_mma_zero(W[1], hi, bh[2], bh[3]);
            lt_mma(W2[0], hi, bl[0], bl[1]);
            lt_mma(W2[1], hi, bl[2], bl[3]);
            const float decay = vec[32];
#pragma unroll
            for (int n = 0; n < 2 * DW; n++)
#pragma unroll
                for (int e = 0; e < 4; e++) S[n][e] *= decay;
            // the warp's eight tokens of the output
            const float4 y = total(2 + part);
            const float2 f = *reinterpret_cast<const float2 *>(vec + 16 + part * 8 + 2 * tq);
            float o[4] = {f.x * y.x, f.y * y.y, f.x * y.z, f.y * y.w}, o2[4], o3[4];
            uint32_t q[4], wh[4], wl[4], kb[DW][4];
            lt_ldmatrix_x4(q, st + b_out);
#pragma unroll
            for (int n = 0; n < 2; n++)
#pragma unroll
                for (int e = 0; e < 4; e++) W[n][e] += W2[n][e];
            split_tile(W, wh, wl);
#pragma unroll
            for (int np = 0; np < DW; np++) {
                lt_ldmatrix_x4_trans(kb[np], st + L.y + b_trans + (uint32_t)np * 32u);
                lt_mma(S[2 * np], wh, kb[np][0], kb[np][1]);
                lt_mma(S[2 * np + 1], wh, kb[np][2], kb[np][3]);
            }
            lt_mma(o, hi, q[0], q[1]);
            lt_mma_zero(o2, lo, q[0], q[1]);
            lt_mma_zero(o3, hi, q[2], q[3]);
#pragma unroll
            for (int np = 0; np < DW; np++) {
                lt_mma(S[2 * np], wl, kb[np][0], kb[np][1]);
                lt_mma(S[2 * np + 1], wl, kb[np][2], kb[np][3]);
            }
            __syncwarp();
            if (lane == 0) mbar_arrive(&empty[sl]);
#pragma unroll
            for (int e = 0; e < 4; e++) o[e] += o2[e] + o3[e];
            const int t = 16 * it + part * 8 + 2 * tq;
            if (t < a.tokens) {
                if (col0) to[0] = o[0];
                if (col1) to[8] = o[2];
            }
            if (t + 1 < a.tokens) {
                if (col0) to[ldv] = o[1];
                if (col1) to[ldv + 8] = o[3];
            }
        }
        if (!ok) atomicExch(&s_failed, 1);
        state_io(true);
    }
    __syncthreads();
    if (tid == 0 && s_failed && a.err) atomicExch(a.err, DEV_ERR_MBAR_TIMEOUT);
}

}  // namespace rnb
