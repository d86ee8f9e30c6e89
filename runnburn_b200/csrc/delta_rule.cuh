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
    const float *conv;         // taps of the q, k and v channels [channels][taps], one after the other
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

// Input of channel c (column `col` of the projections) at token t of this call; t < 0: before it.
template <class AT>
__device__ __forceinline__ float delta_input(const DeltaArgs &a, int c, int col, int t, int pos0) {
    if (t >= 0) return to_f32(reinterpret_cast<const AT *>(a.p)[(size_t)t * a.ld + col]);
    const int pos = pos0 + t, C = 2 * a.kv_heads * a.dim + a.heads * a.vdim;
    return pos >= 0 ? a.ring[(size_t)(pos % delta_ring_rows(a.taps)) * C + c] : 0.f;
}
// column of the projections that channel c comes from
__device__ __forceinline__ int delta_col(const DeltaArgs &a, int c) {
    const int qc = a.kv_heads * a.dim;
    return c < qc ? c : c < 2 * qc ? a.k_at + c - qc : a.v_at + c - 2 * qc;
}
// The inputs that the next call's convolutions reach back to, for channels first, first + step, ... < end
template <class AT>
__device__ __forceinline__ void delta_ring_store(const DeltaArgs &a, int first, int step, int end, int pos0) {
    const int C = 2 * a.kv_heads * a.dim + a.heads * a.vdim, R = delta_ring_rows(a.taps);
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
    const int C = 2 * a.kv_heads * a.dim + a.heads * a.vdim, c = blockIdx.x * 256 + threadIdx.x;
    delta_ring_store<AT>(a, c, C, C, *a.pos0);
}

__host__ inline size_t delta_step_smem(int dim) { return sizeof(float) * (size_t)(DR_BLOCK * (2 * dim + 32) + 3 * DR_BLOCK + 8 * 64); }
// grid = (heads, ceil(vdim / 32)), 256 threads: lane = value column, warp w holds channels w, w + 8, ... (TI of them).
// With act the CTA of a head that finishes last normalises and gates the head's outputs, and the ring is written (tokens <= 8).
template <class AT, int TI>
RNB_GLOBAL void __launch_bounds__(256)
delta_step_kernel(const __grid_constant__ DeltaArgs a) {
    extern __shared__ __align__(16) float ds_smem[];
    pdl_launch_dependents();
    const int dim = a.dim, vdim = a.vdim, h = blockIdx.x, j0 = blockIdx.y * 32, rep = a.heads / a.kv_heads, hk = h / rep;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, j = j0 + lane, qc = a.kv_heads * dim;
    const bool live = j < vdim;
    float *sq = ds_smem, *sk = sq + DR_BLOCK * dim, *sv = sk + DR_BLOCK * dim, *sg = sv + DR_BLOCK * 32, *sb = sg + DR_BLOCK, *sqk = sb + DR_BLOCK, *red = sqk + DR_BLOCK;
    float *sp = a.state + (size_t)h * dim * vdim + j;
    if (vdim >= 32) {
        for (int ch = tid; ch < dim; ch += 256) asm volatile("prefetch.global.L2 [%0];" ::"l"(a.state + ((size_t)h * dim + ch) * vdim + j0));
    } else {
        prefetch_l2(a.state + (size_t)h * dim * vdim, (size_t)dim * vdim * 4, tid, 256);
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
                for (int n = 0; n < a.taps; n++) y = fmaf(a.conv[(size_t)c * a.taps + n], delta_input<AT>(a, c, col, t0 + t - (a.taps - 1) + n, pos0), y);
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
    if (h % rep == 0 && blockIdx.y == 0) {
        delta_ring_store<AT>(a, hk * dim + tid, 256, (hk + 1) * dim, pos0);
        delta_ring_store<AT>(a, qc + hk * dim + tid, 256, qc + (hk + 1) * dim, pos0);
    }
    if (tid < 32) delta_ring_store<AT>(a, 2 * qc + h * vdim + j, 32, 2 * qc + h * vdim + min(j0 + 32, vdim), pos0);
    if (last_of_head(a.counters + h, gridDim.y))
        head_norm_gate_rows(a.o, reinterpret_cast<const float *>(a.p) + a.g_at, a.norm, a.act, a.tokens, a.heads, h, vdim, 0, a.ld, a.lda, a.eps, a.out_mul);
}

// ---- prompts on tensor cores ---------------------------------------------------------------------
// Record of a tile and head: T beta (bf16 hi, lo), P (hi, lo): 16 x 16 each, row t, column s; then f32: G_t0 a_t [16],
// G_t0 b_t [16], G_Tt a_t [16], G_T0 [1].
constexpr int DR_MAT = 16 * 16 * 2, DR_VEC = 4 * DR_MAT, DR_REC = DR_VEC + 4 * 64;
__host__ __device__ inline size_t delta_prepare_smem(int dim) { return (size_t)2 * 16 * (dim + 8) * 2 + (2 * 16 * 17 + 32) * 4 + 8 * (16 * 17 + 32) * 4; }

// grid = (ceil(tokens / 16), kv_heads), 256 threads.  dim and vdim multiples of 8, dim of 16.
RNB_GLOBAL void __launch_bounds__(256)
delta_prepare_kernel(const __grid_constant__ DeltaArgs a) {
    extern __shared__ __align__(16) uint8_t dp_smem[];
    pdl_launch_dependents();
    pdl_wait();
    const int dim = a.dim, rep = a.heads / a.kv_heads, hk = blockIdx.y, t0 = blockIdx.x * 16, nt = min(16, a.tokens - t0), pos0 = *a.pos0;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, KE = dim + 8, qc = a.kv_heads * dim;
    bf16 *sx = reinterpret_cast<bf16 *>(dp_smem), *sy = sx + 16 * KE;
    float *xy = reinterpret_cast<float *>(sy + 16 * KE), *yy = xy + 16 * 17, *nrm = yy + 16 * 17, *wrk = nrm + 32 + warp * (16 * 17 + 32);
    const bf16 *p = reinterpret_cast<const bf16 *>(a.p);
    // convolutions: 8 channels of 4 tokens at a time; rows past the end become zeros
    const int units = (2 * dim + rep * a.vdim) / 8;
    for (int i = tid; i < units * 4; i += 256) {
        const int u = i % units, ts = i / units * 4, x = u * 8;
        const int c = x < dim ? hk * dim + x : x < 2 * dim ? qc + hk * dim + x - dim : 2 * qc + hk * rep * a.vdim + x - 2 * dim;
        const int col = delta_col(a, c);
        float y[4][8] = {};
        for (int n = 0; n < a.taps; n++) {
            float w[8];
#pragma unroll
            for (int e = 0; e < 8; e++) w[e] = a.conv[(size_t)(c + e) * a.taps + n];
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
    for (int i = warp; i < 32; i += 8) {   // inverse norms: queries 0..15, keys 16..31
        const bf16 *r = i < 16 ? sx + i * KE : sy + (i - 16) * KE;
        float s = 0.f;
        for (int ch = lane; ch < dim; ch += 32) s = fmaf(to_f32(r[ch]), to_f32(r[ch]), s);
        s = warp_sum(s);
        if (lane == 0) nrm[i] = (i < 16 ? a.q_mul : 1.0f) / sqrtf(s + DR_UNIT_EPS);
    }
    const int g = lane >> 2, tq = lane & 3, mi = lane >> 3, mr = lane & 7;
    if (warp < 2) {   // x y^T, y y^T
        float s[2][4] = {};
        const uint32_t pitch = (uint32_t)KE * 2, am = smem_u32(warp ? sy : sx) + (uint32_t)((mi & 1) * 8 + mr) * pitch + (uint32_t)(mi >> 1) * 16u;
        const uint32_t bm = smem_u32(sy) + (uint32_t)((mi >> 1) * 8 + mr) * pitch + (uint32_t)(mi & 1) * 16u;
        for (int ks = 0; ks < dim / 16; ks++) {
            uint32_t fa[4], fb[4];
            lt_ldmatrix_x4(fa, am + (uint32_t)ks * 32u);
            lt_ldmatrix_x4(fb, bm + (uint32_t)ks * 32u);
            lt_mma(s[0], fa, fb[0], fb[1]);
            lt_mma(s[1], fa, fb[2], fb[3]);
        }
        float *out = warp ? yy : xy;
#pragma unroll
        for (int n = 0; n < 2; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) out[(g + 8 * (e >> 1)) * 17 + n * 8 + 2 * tq + (e & 1)] = s[n][e];
    }
    __syncthreads();
    // a warp per head; lane s = column s of the matrices
    float *M = wrk, *lg = wrk + 16 * 17, *bt = lg + 16;
    const int s = lane & 15;
    for (int r = warp; r < rep; r += 8) {
        const int h = hk * rep + r;
        if (lane < 16) {
            const float *ba = a.ba + (size_t)(t0 + min(s, nt - 1)) * a.ld_ba;
            lg[s] = s < nt ? -expf(a.a_log[h]) * softplus_f32(ba[a.a_at + h] + a.dt[h]) : 0.f;
            bt[s] = s < nt ? sigmoid_f32(ba[h]) : 0.f;
        }
        __syncwarp();
        uint8_t *rec = a.rec + ((size_t)blockIdx.x * a.heads + h) * DR_REC;
        bf16 *Thi = reinterpret_cast<bf16 *>(rec), *Tlo = Thi + 256, *Phi = Tlo + 256, *Plo = Phi + 256;
        float *vec = reinterpret_cast<float *>(rec + DR_VEC);
        if (lane < 16) {
            float acc = 0.f, head = 0.f;   // logarithms of G_ts, and of G_s0
            for (int t = 0; t <= s; t++) head += lg[t];
            for (int t = 0; t < 16; t++) {
                if (t > s) acc += lg[t];
                const float e = t >= s ? expf(acc) * nrm[16 + s] : 0.f;
                M[t * 17 + s] = t > s ? bt[t] * nrm[16 + t] * e * yy[t * 17 + s] : 0.f;
                lt_split_store(Phi + t * 16 + s, Plo + t * 16 + s, nrm[t] * e * xy[t * 17 + s]);
            }
            const float from0 = expf(head);
            vec[s] = from0 * nrm[16 + s];
            vec[16 + s] = from0 * nrm[s];
            vec[32 + s] = expf(acc) * nrm[16 + s];
            if (s == 15) vec[48] = from0;
        }
        __syncwarp();
        if (lane < 16) {   // column s of (I + M)^-1 by forward substitution
            float x[16];
#pragma unroll
            for (int t = 0; t < 16; t++) {
                float v = t == s ? 1.f : 0.f;
#pragma unroll
                for (int q = 0; q < 16; q++)
                    if (q < t) v = fmaf(-M[t * 17 + q], x[q], v);
                x[t] = v;
                lt_split_store(Thi + t * 16 + s, Tlo + t * 16 + s, v * bt[s]);
            }
        }
        __syncwarp();
    }
}

constexpr int DT_STAGES = 4;
struct DeltaTileSmem {
    uint32_t kp, vp, y, v, mat, vec, stage, bytes;
};
__host__ __device__ inline DeltaTileSmem delta_tile_smem(int DT, int NW) {
    DeltaTileSmem s;
    s.kp = (uint32_t)(16 * DT + 8) * 2;
    s.vp = (uint32_t)(16 * NW + 8) * 2;
    s.y = 16 * s.kp;                 // x at 0
    s.v = s.y + 16 * s.kp;
    s.mat = s.v + 16 * s.vp;         // four matrices, rows of 48 bytes
    s.vec = s.mat + 4 * 16 * 48;
    s.stage = s.vec + 256;
    s.bytes = DT_STAGES * s.stage;
    return s;
}
// grid = (heads, column blocks), blockDim = 32 * NW: warp w holds S^T of 16 value columns.  dim <= 16 DT a multiple of 16, vdim of 8.
template <int DT>
RNB_GLOBAL void __launch_bounds__(256)
delta_tile_kernel(const __grid_constant__ DeltaArgs a) {
    extern __shared__ __align__(128) uint8_t dt_smem[];
    pdl_launch_dependents();
    pdl_wait();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nthr = blockDim.x, NW = nthr >> 5;
    const DeltaTileSmem L = delta_tile_smem(DT, NW);
    const uint32_t base = smem_u32(dt_smem);
    const int h = blockIdx.x, j0 = blockIdx.y * 16 * NW, hk = h / (a.heads / a.kv_heads), n_tiles = (a.tokens + 15) / 16, vdim = a.vdim;
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
            for (int x = tid; x < 16 * 2 * NW; x += nthr) {
                const int t = x / (2 * NW), q = x % (2 * NW), col = j0 + q * 8;
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
    const int g = lane >> 2, tq = lane & 3, mi = lane >> 3, mr = lane & 7, jw = j0 + warp * 16;
    float S[2 * DT][4];
    auto state_io = [&](bool store) {
#pragma unroll
        for (int n = 0; n < 2 * DT; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int ch = n * 8 + 2 * tq + (e & 1), j = jw + g + 8 * (e >> 1);
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
    const uint32_t b_plain = (uint32_t)((mi >> 1) * 8 + mr) * L.kp + (uint32_t)(mi & 1) * 16u;        // rows (n), k contiguous
    const uint32_t b_trans = (uint32_t)((mi & 1) * 8 + mr) * L.kp + (uint32_t)(mi >> 1) * 16u;        // rows (k), n contiguous
    const uint32_t b_mat = (uint32_t)((mi >> 1) * 8 + mr) * 48u + (uint32_t)(mi & 1) * 16u;
    for (int it = 0; it < n_tiles; it++) {
        asm volatile("cp.async.wait_group %0;" ::"n"(DT_STAGES - 2) : "memory");
        __syncthreads();   // the tile is in, and every warp is through with the one whose stage is loaded next
        load_tile(it + DT_STAGES - 1);
        const uint32_t st = base + (uint32_t)(it % DT_STAGES) * L.stage;
        const uint8_t *raw = dt_smem + (size_t)(it % DT_STAGES) * L.stage;
        const float *vec = reinterpret_cast<const float *>(raw + L.vec);
        // (S0^T y, S0^T x): state hi + lo, exact bf16 rows
        float X[4][4] = {}, Y[4][4] = {};
#pragma unroll
        for (int ks = 0; ks < DT; ks++) {
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
        // V - G_t0 a_t S0^T y
        const bf16 *sv = reinterpret_cast<const bf16 *>(raw + L.v);
        const int VE = (int)(L.vp / 2);
        float R[2][4];
#pragma unroll
        for (int n = 0; n < 2; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int t = n * 8 + 2 * tq + (e & 1);
                R[n][e] = to_f32(sv[t * VE + warp * 16 + g + 8 * (e >> 1)]) - vec[t] * (X[n][e] + X[n + 2][e]);
            }
        auto split_tile = [&](const float (&m)[2][4], uint32_t (&hi)[4], uint32_t (&lo)[4]) {
            lt_split(m[0][0], m[0][1], hi[0], lo[0]);
            lt_split(m[0][2], m[0][3], hi[1], lo[1]);
            lt_split(m[1][0], m[1][1], hi[2], lo[2]);
            lt_split(m[1][2], m[1][3], hi[3], lo[3]);
        };
        auto times = [&](float (&o)[2][4], const uint32_t (&hi)[4], const uint32_t (&lo)[4], uint32_t mat) {
            uint32_t bh[4], bl[4];
            lt_ldmatrix_x4(bh, st + L.mat + mat + b_mat);
            lt_ldmatrix_x4(bl, st + L.mat + mat + 16 * 48 + b_mat);
            lt_mma(o[0], hi, bh[0], bh[1]);
            lt_mma(o[1], hi, bh[2], bh[3]);
            lt_mma(o[0], lo, bh[0], bh[1]);
            lt_mma(o[1], lo, bh[2], bh[3]);
            lt_mma(o[0], hi, bl[0], bl[1]);
            lt_mma(o[1], hi, bl[2], bl[3]);
        };
        uint32_t hi[4], lo[4];
        float U[2][4] = {}, O[2][4], W[2][4];
        split_tile(R, hi, lo);
        times(U, hi, lo, 0);
#pragma unroll
        for (int n = 0; n < 2; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int t = n * 8 + 2 * tq + (e & 1);
                W[n][e] = U[n][e] * vec[32 + t];
                O[n][e] = vec[16 + t] * (Y[n][e] + Y[n + 2][e]);
            }
        // the state moves on first: the next tile waits for it
        uint32_t wh[4], wl[4];
        split_tile(W, wh, wl);
        const float decay = vec[48];
#pragma unroll
        for (int np = 0; np < DT; np++) {
            uint32_t kb[4];
            lt_ldmatrix_x4_trans(kb, st + L.y + b_trans + (uint32_t)np * 32u);
#pragma unroll
            for (int e = 0; e < 4; e++) S[2 * np][e] *= decay, S[2 * np + 1][e] *= decay;
            lt_mma(S[2 * np], wh, kb[0], kb[1]);
            lt_mma(S[2 * np + 1], wh, kb[2], kb[3]);
            lt_mma(S[2 * np], wl, kb[0], kb[1]);
            lt_mma(S[2 * np + 1], wl, kb[2], kb[3]);
        }
        split_tile(U, hi, lo);
        times(O, hi, lo, 2 * 16 * 48);
#pragma unroll
        for (int n = 0; n < 2; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int t = 16 * it + n * 8 + 2 * tq + (e & 1), j = jw + g + 8 * (e >> 1);
                if (t < a.tokens && j < vdim) a.o[((size_t)t * a.heads + h) * vdim + j] = O[n][e];
            }
    }
    state_io(true);
}

}  // namespace rnb
