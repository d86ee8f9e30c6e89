// Linear recurrences with a matrix state per head (RWKV-style time mixing, retention, gated linear
// attention), all in f32:
//   o_t = rs * S^T r_t + (sum_i r_t[i] u[i] k_t[i]) v_t,      S <- diag(w_t) S + k_t v_t^T
// Time mixing: w_t per key channel, u the bonus of the current token, rs = 1.  Retention, whose output
// reads the updated state S_t = decay S + k v^T: w_t = decay of the head, u = 1, rs = decay.  Gated linear
// attention reads the updated state too, with w_t per key channel: the first term takes w_t r_t, u = 1.
// State [heads][dim][vdim] f32.
//
//   linear_state_step_kernel    1..8 tokens, one launch: rotations or decays, recurrence, head norm, gate
//   linear_state_chunk_kernel   many tokens: the sequence is cut into chunks that run at the same time.
//       OUT = false: every chunk but the last accumulates its own contribution from a zero state;
//       linear_state_scan_kernel turns these into the state at the start of every chunk;
//       OUT = true: every chunk runs again from its start state and writes its outputs.
//   linear_state_tile_kernel    the same two passes on tensor cores for bf16 projections: 16 tokens at a time
//     (the state stays in f32 accumulators and enters products as bf16 hi + lo parts).
//   Decays enter as products of w, never as ratios of products: nothing can overflow.
#pragma once
#include "layer_glue.cuh"
#include "mma_bf16.cuh"

namespace rnb {

enum LinearMode { LS_BONUS = 0, LS_HEAD_DECAY = 1, LS_UPDATED = 2 };   // time mixing, retention, gated linear attention
struct LinearChunkArgs {
    const void *r, *k, *v;     // [tokens][heads][dim], same, [tokens][heads][vdim] (AT); a token's row is ldr (r, k), ldv long
    const float *w;            // [tokens][heads][dim]; LS_HEAD_DECAY: decay[head] instead
    const float *decay, *u;    // [heads]; [heads][dim], null: 1
    float o_mul;               // multiplies the outputs
    float *state, *o;          // [heads][dim][vdim]; [tokens][heads][vdim]
    float *starts, *decays;    // [chunks][heads][dim][vdim]; [chunks][heads][dim]
    int tokens, heads, dim, vdim, ldr, ldv, chunk, n_chunks;
    int G, JG;                 // lanes along dim (16 channels each), groups of 4 value columns per CTA
};
constexpr int LS_TI = 16, LS_TS = 16;   // channels per thread; tokens staged at a time
__host__ __device__ inline size_t linear_chunk_smem(int G, int JG) { return sizeof(float) * ((size_t)LS_TS * (3 * LS_TI * G + 4 * JG) + LS_TS); }

// grid = (chunks, heads, column blocks); G * JG threads rounded up to a warp.
// Thread (jg, g): value columns 4 jg .. + 3, channels 4 (q G + g) .. + 3 for q = 0..3.
template <class AT, bool OUT, int MODE>
RNB_GLOBAL void __launch_bounds__(256)
linear_state_chunk_kernel(const __grid_constant__ LinearChunkArgs a) {
    constexpr bool CONST_W = MODE == LS_HEAD_DECAY;
    extern __shared__ __align__(16) float ls_smem[];
    pdl_launch_dependents();
    pdl_wait();
    const int G = a.G, DP = LS_TI * G, VB = 4 * a.JG;
    float *sr = ls_smem, *sk = sr + LS_TS * DP, *sw = sk + LS_TS * DP, *sv = sw + LS_TS * DP, *sb = sv + LS_TS * VB;
    const int c = blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * VB, tid = threadIdx.x;
    const int g = tid & (G - 1), jg = tid / G, j = j0 + 4 * jg;
    const bool live = jg < a.JG;
    const int t_begin = c * a.chunk, t_end = min(t_begin + a.chunk, a.tokens);
    const float cw = CONST_W ? a.decay[h] : 1.f, rs = CONST_W ? cw : 1.f;
    const AT *rp = reinterpret_cast<const AT *>(a.r), *kp = reinterpret_cast<const AT *>(a.k), *vp = reinterpret_cast<const AT *>(a.v);
    float S[LS_TI][4], P[LS_TI];
#pragma unroll
    for (int i = 0; i < LS_TI; i++) {
        P[i] = 1.f;
#pragma unroll
        for (int e = 0; e < 4; e++) S[i][e] = 0.f;
    }
    auto state_io = [&](float *base, bool store) {
        if (!live) return;
#pragma unroll
        for (int i = 0; i < LS_TI; i++) {
            const int ch = 4 * ((i >> 2) * G + g) + (i & 3);
            if (ch >= a.dim) continue;
            float *p = base + ((size_t)h * a.dim + ch) * a.vdim + j;
#pragma unroll
            for (int e = 0; e < 4; e++)
                if (j + e < a.vdim) {
                    if (store) p[e] = S[i][e];
                    else S[i][e] = p[e];
                }
        }
    };
    const size_t cs = (size_t)a.heads * a.dim * a.vdim;
    if (OUT) state_io(a.n_chunks > 1 ? a.starts + (size_t)c * cs : a.state, false);
    for (int t0 = t_begin; t0 < t_end; t0 += LS_TS) {
        const int nt = min(LS_TS, t_end - t0);
        __syncthreads();
        for (int i = tid; i < nt * DP; i += blockDim.x) {
            const int t = i / DP, ch = i % DP;
            const bool in = ch < a.dim;
            const size_t at = (size_t)(t0 + t) * a.ldr + h * a.dim + ch;
            if (OUT) sr[i] = in ? to_f32(rp[at]) : 0.f;
            sk[i] = in ? to_f32(kp[at]) : 0.f;
            if (!CONST_W) sw[i] = in ? a.w[((size_t)(t0 + t) * a.heads + h) * a.dim + ch] : 0.f;
        }
        for (int i = tid; i < nt * VB; i += blockDim.x) {
            const int t = i / VB, col = j0 + i % VB;
            sv[i] = col < a.vdim ? to_f32(vp[(size_t)(t0 + t) * a.ldv + h * a.vdim + col]) : 0.f;
        }
        __syncthreads();
        if (OUT) {
            for (int t = tid >> 5; t < nt; t += blockDim.x >> 5) {
                float b = 0.f;
                for (int ch = tid & 31; ch < a.dim; ch += 32) b = fmaf(sr[t * DP + ch] * (a.u ? a.u[h * a.dim + ch] : 1.f), sk[t * DP + ch], b);
                b = warp_sum(b);
                if ((tid & 31) == 0) sb[t] = b;
            }
            __syncthreads();
        }
        for (int t = 0; t < nt; t++) {
            const float4 v4 = live ? *reinterpret_cast<const float4 *>(sv + t * VB + 4 * jg) : make_float4(0.f, 0.f, 0.f, 0.f);
            const float vv[4] = {v4.x, v4.y, v4.z, v4.w};
            float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int q = 0; q < LS_TI / 4; q++) {
                const int at = t * DP + 4 * (q * G + g);
                const float4 k4 = *reinterpret_cast<const float4 *>(sk + at);
                const float kk[4] = {k4.x, k4.y, k4.z, k4.w};
                float rr[4], ww[4];
                if (OUT) {
                    const float4 r4 = *reinterpret_cast<const float4 *>(sr + at);
                    rr[0] = r4.x, rr[1] = r4.y, rr[2] = r4.z, rr[3] = r4.w;
                }
                if (CONST_W) {
                    ww[0] = ww[1] = ww[2] = ww[3] = cw;
                } else {
                    const float4 w4 = *reinterpret_cast<const float4 *>(sw + at);
                    ww[0] = w4.x, ww[1] = w4.y, ww[2] = w4.z, ww[3] = w4.w;
                }
#pragma unroll
                for (int i = 0; i < 4; i++) {
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        if (OUT) acc[e] = fmaf(MODE == LS_UPDATED ? rr[i] * ww[i] : rr[i], S[4 * q + i][e], acc[e]);
                        S[4 * q + i][e] = fmaf(ww[i], S[4 * q + i][e], kk[i] * vv[e]);
                    }
                    if (!OUT && !CONST_W) P[4 * q + i] *= ww[i];
                }
            }
            if (OUT) {
                for (int d = 1; d < G; d <<= 1) {
#pragma unroll
                    for (int e = 0; e < 4; e++) acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], d);
                }
                if (live && g == 0) {
                    float *o = a.o + ((size_t)(t0 + t) * a.heads + h) * a.vdim + j;
#pragma unroll
                    for (int e = 0; e < 4; e++)
                        if (j + e < a.vdim) o[e] = fmaf(rs, acc[e], sb[t] * vv[e]) * a.o_mul;
                }
            }
        }
    }
    if (OUT) {
        if (c == a.n_chunks - 1) state_io(a.state, true);
    } else {
        state_io(a.starts + (size_t)c * cs, true);
        if (!CONST_W && blockIdx.z == 0 && jg == 0)
#pragma unroll
            for (int i = 0; i < LS_TI; i++) {
                const int ch = 4 * ((i >> 2) * G + g) + (i & 3);
                if (ch < a.dim) a.decays[((size_t)c * a.heads + h) * a.dim + ch] = P[i];
            }
    }
}

// starts[c] <- the state at the start of chunk c, from the chunks' own contributions.  One thread per V state
// elements of a channel's row; the contributions of eight chunks are in flight at a time.
template <int V>
RNB_GLOBAL void __launch_bounds__(256)
linear_state_scan_kernel(const float *__restrict__ state, float *starts, const float *__restrict__ decays, const float *__restrict__ decay, int heads, int dim,
                         int vdim, int chunk, int n_chunks) {
    pdl_launch_dependents();
    pdl_wait();
    struct alignas(4 * V) Vec { float v[V]; };
    const size_t n = (size_t)heads * dim * vdim, i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * V;
    if (i >= n) return;
    const size_t row = i / vdim, rows = (size_t)heads * dim;
    Vec S = *reinterpret_cast<const Vec *>(state + i);
    const float p0 = decays ? 0.f : powf(decay[row / dim], (float)chunk);
    for (int c0 = 0; c0 < n_chunks - 1; c0 += 8) {
        Vec add[8];
        float p[8];
#pragma unroll
        for (int q = 0; q < 8; q++)
            if (c0 + q < n_chunks - 1) {
                add[q] = *reinterpret_cast<const Vec *>(starts + (size_t)(c0 + q) * n + i);
                p[q] = decays ? decays[(size_t)(c0 + q) * rows + row] : p0;
            }
#pragma unroll
        for (int q = 0; q < 8; q++)
            if (c0 + q < n_chunks - 1) {
                *reinterpret_cast<Vec *>(starts + (size_t)(c0 + q) * n + i) = S;
#pragma unroll
                for (int e = 0; e < V; e++) S.v[e] = fmaf(p[q], S.v[e], add[q].v[e]);
            }
    }
    *reinterpret_cast<Vec *>(starts + (size_t)(n_chunks - 1) * n + i) = S;
}

// Decays from their low-rank input: out[t][c] = decay_of(sum_j w2[c][j] f(z[t][j]) + w0[c]); f: tanh for DECAY_EXP, else none.
// grid = (ceil(channels / 128), ceil(tokens / 16)), 128 threads; dynamic shared memory 16 * rank floats.
RNB_GLOBAL void __launch_bounds__(128)
decay_rows_kernel(const float *__restrict__ z, const bf16 *__restrict__ w2, const float *__restrict__ w0, int tokens, int rank, int channels, int kind,
                  float inv_tau, float *__restrict__ out) {
    extern __shared__ __align__(16) float dr_smem[];   // [rank][16]
    pdl_launch_dependents();
    pdl_wait();
    const int t0 = blockIdx.y * 16;
    for (int i = threadIdx.x; i < rank * 16; i += blockDim.x) {
        const int t = i / rank, j = i % rank;
        const float v = t0 + t < tokens ? z[(size_t)(t0 + t) * rank + j] : 0.f;
        dr_smem[j * 16 + t] = kind == DECAY_EXP ? tanhf(v) : v;
    }
    __syncthreads();
    const int c = blockIdx.x * 128 + threadIdx.x;
    if (c >= channels) return;
    float acc[16];
    const float b = w0[c];
#pragma unroll
    for (int t = 0; t < 16; t++) acc[t] = 0.f;
    for (int j = 0; j < rank; j++) {
        const float w = to_f32(w2[(size_t)c * rank + j]);
#pragma unroll
        for (int q = 0; q < 4; q++) {
            const float4 v = *reinterpret_cast<const float4 *>(dr_smem + j * 16 + 4 * q);
            acc[4 * q] = fmaf(w, v.x, acc[4 * q]);
            acc[4 * q + 1] = fmaf(w, v.y, acc[4 * q + 1]);
            acc[4 * q + 2] = fmaf(w, v.z, acc[4 * q + 2]);
            acc[4 * q + 3] = fmaf(w, v.w, acc[4 * q + 3]);
        }
    }
#pragma unroll
    for (int t = 0; t < 16; t++)
        if (t0 + t < tokens) out[(size_t)(t0 + t) * channels + c] = decay_of(kind, acc[t] + b, inv_tau);
}

// z [tokens][rank] f32 -> [f(z) rounded to bf16 | what the rounding left] [tokens][2 rank], f = tanh or none: against
// [w2 | w2] the tensor-core matmul gives w2 f(z) to about f32 accuracy.
RNB_GLOBAL void __launch_bounds__(256)
split_rows_kernel(const float *__restrict__ z, int rank, size_t n, int kind, bf16 *__restrict__ out) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    const float v = kind == DECAY_EXP ? tanhf(z[i]) : z[i];
    const bf16 hi = from_f32<bf16>(v);
    bf16 *row = out + (i / rank) * 2 * rank + i % rank;
    row[0] = hi;
    row[rank] = from_f32<bf16>(v - to_f32(hi));
}

// ---- many tokens on tensor cores -----------------------------------------------------------------
// Shared memory of a CTA of NW warps (16 value columns each): two stages of raw rows, then the processed ones.
struct LinearTileSmem {
    uint32_t kp, vp, stage, k, w, v, rhi, rlo, khi, klo, ahi, alo, d, p, pw, bytes;
};
__host__ __device__ inline LinearTileSmem linear_tile_smem(int DT, int NW) {
    LinearTileSmem s;
    s.kp = (uint32_t)(16 * DT + 8) * 2;
    s.vp = (uint32_t)(16 * NW + 8) * 2;
    s.k = 16 * s.kp;
    s.w = s.k + 16 * s.kp;
    s.v = s.w + 16 * 16 * DT * 4;
    s.stage = s.v + 16 * s.vp;
    s.rhi = 2 * s.stage;
    s.rlo = s.rhi + 16 * s.kp;
    s.khi = s.rlo + 16 * s.kp;
    s.klo = s.khi + 16 * s.kp;
    s.ahi = s.klo + 16 * s.kp;
    s.alo = s.ahi + 16 * 48;
    s.d = s.alo + 16 * 48;
    s.p = s.d + 16 * DT * 4;
    s.pw = s.p + 16 * DT * 4;
    s.bytes = s.pw + 32 * 4;
    return s;
}
// Per tile of 16 tokens, with S^T (value column x channel) in each warp's accumulators:
//   o^T = S^T r~^T + v^T A^T          r~_t = r_t times the decays before t,  A: pairs inside the tile
//   S^T <- S^T D + v^T k~             k~_t = k_t times the decays after t,   D: all decays of the tile
// (gated linear attention: r~_t takes the decay of t itself too, and so do the pairs of A)
// Time mixing computes A below the diagonal pair by pair (running products of w), with r u k on it;
// retention masks and scales q k^T by powers of its decay, and scales S^T q^T by them afterwards.
// grid = (chunks, heads, column blocks), blockDim = 32 * NW.  dim <= 16 DT, dim and vdim multiples of 8.
template <int DT, bool OUT, int MODE>
RNB_GLOBAL void __launch_bounds__(256)
linear_state_tile_kernel(const __grid_constant__ LinearChunkArgs a) {
    constexpr bool CONST_W = MODE == LS_HEAD_DECAY;
    extern __shared__ __align__(128) uint8_t lt_smem[];
    pdl_launch_dependents();
    pdl_wait();
    constexpr int DP = 16 * DT;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nthr = blockDim.x, NW = nthr >> 5;
    const LinearTileSmem L = linear_tile_smem(DT, NW);
    const uint32_t base = smem_u32(lt_smem);
    const int c = blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * 16 * NW;
    const int t_begin = c * a.chunk, t_end = min(t_begin + a.chunk, a.tokens), n_tiles = (t_end - t_begin + 15) / 16;
    const bf16 *rp = reinterpret_cast<const bf16 *>(a.r) + (size_t)h * a.dim, *kp = reinterpret_cast<const bf16 *>(a.k) + (size_t)h * a.dim;
    const bf16 *vp = reinterpret_cast<const bf16 *>(a.v) + (size_t)h * a.vdim;
    const float *wp = CONST_W ? nullptr : a.w + (size_t)h * a.dim;
    const size_t ldk = (size_t)a.ldr, ldw = (size_t)a.heads * a.dim, ldv = (size_t)a.ldv;
    float *sD = reinterpret_cast<float *>(lt_smem + L.d), *sP = reinterpret_cast<float *>(lt_smem + L.p), *pw = reinterpret_cast<float *>(lt_smem + L.pw);
    auto cp16 = [&](uint32_t dst, const void *src, bool in) {
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(in ? 16u : 0u) : "memory");
    };
    auto load_tile = [&](int i) {
        const uint32_t st = base + (uint32_t)(i & 1) * L.stage;
        const int t0 = t_begin + 16 * i;
        constexpr int CK = DP / 8, CWF = DP / 4;
        // eight threads walk along a row; 256 threads put two such groups on each row
        const int groups = nthr == 256 ? 2 : 1, q0 = (tid & 7) + (groups == 2 ? 8 * (tid >> 7) : 0), qs = 8 * groups;
        for (int t = (groups == 2 ? tid & 127 : tid) >> 3; t < 16; t += nthr / (8 * groups)) {
            const int tok = t0 + t;
            const size_t row = (size_t)min(tok, t_end - 1);
            const bool in = tok < t_end;
            for (int q = q0; q < CK; q += qs) {
                const bool ok = in && q * 8 < a.dim;
                const int at = min(q * 8, a.dim - 8);
                cp16(st + L.k + (uint32_t)t * L.kp + (uint32_t)q * 16u, kp + row * ldk + at, ok);
                if (OUT) cp16(st + (uint32_t)t * L.kp + (uint32_t)q * 16u, rp + row * ldk + at, ok);
            }
            if (!CONST_W)
                for (int q = q0; q < CWF; q += qs) cp16(st + L.w + (uint32_t)(t * DP + q * 4) * 4u, wp + row * ldw + min(q * 4, a.dim - 4), in && q * 4 < a.dim);
            for (int q = q0; q < 2 * NW; q += qs) {
                const int col = j0 + q * 8;
                cp16(st + L.v + (uint32_t)t * L.vp + (uint32_t)q * 16u, vp + row * ldv + min(col, a.vdim - 8), in && col < a.vdim);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load_tile(0);
    const float cw = CONST_W ? a.decay[h] : 1.f;
    if (CONST_W && tid <= 16) pw[tid] = powf(cw, (float)tid);
    if (!OUT && !CONST_W)
        for (int i = tid; i < DP; i += nthr) sP[i] = 1.f;
    const int g = lane >> 2, tq = lane & 3, mi = lane >> 3, mr = lane & 7, jw = j0 + warp * 16;
    float S[2 * DT][4];
    const size_t cs = (size_t)a.heads * a.dim * a.vdim;
    auto state_io = [&](float *b, bool store) {
#pragma unroll
        for (int n = 0; n < 2 * DT; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int ch = n * 8 + 2 * tq + (e & 1), j = jw + g + 8 * (e >> 1);
                const bool in = ch < a.dim && j < a.vdim;
                float *p = b + ((size_t)h * a.dim + ch) * a.vdim + j;
                if (store) {
                    if (in) *p = S[n][e];
                } else {
                    S[n][e] = in ? *p : 0.f;
                }
            }
    };
    if (OUT) state_io(a.n_chunks > 1 ? a.starts + (size_t)c * cs : a.state, false);
    else
#pragma unroll
        for (int n = 0; n < 2 * DT; n++) S[n][0] = S[n][1] = S[n][2] = S[n][3] = 0.f;
    // fragment addresses that do not change from tile to tile
    const uint32_t b_plain = (uint32_t)((mi >> 1) * 8 + mr) * L.kp + (uint32_t)(mi & 1) * 16u;        // rows (n), k contiguous
    const uint32_t b_trans = (uint32_t)((mi & 1) * 8 + mr) * L.kp + (uint32_t)(mi >> 1) * 16u;        // rows (k), n contiguous
    for (int it = 0; it < n_tiles; it++) {
        if (it + 1 < n_tiles) {
            load_tile(it + 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();   // raw rows are in; the previous tile's processed rows are free
        uint8_t *raw = lt_smem + (size_t)(it & 1) * L.stage;
        const int t0 = t_begin + 16 * it, nt = min(16, t_end - t0);
        const bf16 *rr = reinterpret_cast<const bf16 *>(raw), *kk = reinterpret_cast<const bf16 *>(raw + L.k);
        const float *ww = reinterpret_cast<const float *>(raw + L.w);
        bf16 *rhi = reinterpret_cast<bf16 *>(lt_smem + L.rhi), *rlo = reinterpret_cast<bf16 *>(lt_smem + L.rlo);
        bf16 *khi = reinterpret_cast<bf16 *>(lt_smem + L.khi), *klo = reinterpret_cast<bf16 *>(lt_smem + L.klo);
        bf16 *ahi = reinterpret_cast<bf16 *>(lt_smem + L.ahi), *alo = reinterpret_cast<bf16 *>(lt_smem + L.alo);
        constexpr int KE = DP + 8;
        if (CONST_W) {
            for (int x = tid; x < 16 * (DP / 8); x += nthr) {
                const int t = x / (DP / 8), at = t * KE + x % (DP / 8) * 8;
                const uint4 b = *reinterpret_cast<const uint4 *>(kk + at);
                const float p = t < nt ? pw[nt - 1 - t] : 0.f;
                uint4 hi, lo;
                lt_split(bf16_lo(b.x) * p, bf16_hi(b.x) * p, hi.x, lo.x);
                lt_split(bf16_lo(b.y) * p, bf16_hi(b.y) * p, hi.y, lo.y);
                lt_split(bf16_lo(b.z) * p, bf16_hi(b.z) * p, hi.z, lo.z);
                lt_split(bf16_lo(b.w) * p, bf16_hi(b.w) * p, hi.w, lo.w);
                *reinterpret_cast<uint4 *>(khi + at) = hi;
                *reinterpret_cast<uint4 *>(klo + at) = lo;
            }
            if (OUT && warp == 0) {
                float q[2][4] = {};
                const uint32_t ra = base + (uint32_t)(it & 1) * L.stage + (uint32_t)((mi & 1) * 8 + mr) * L.kp + (uint32_t)(mi >> 1) * 16u;
                const uint32_t kb = base + (uint32_t)(it & 1) * L.stage + L.k + b_plain;
#pragma unroll
                for (int ks = 0; ks < DT; ks++) {
                    uint32_t ra4[4], kb4[4];
                    lt_ldmatrix_x4(ra4, ra + (uint32_t)ks * 32u);
                    lt_ldmatrix_x4(kb4, kb + (uint32_t)ks * 32u);
                    lt_mma(q[0], ra4, kb4[0], kb4[1]);
                    lt_mma(q[1], ra4, kb4[2], kb4[3]);
                }
#pragma unroll
                for (int n = 0; n < 2; n++)
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        const int t = g + 8 * (e >> 1), s = n * 8 + 2 * tq + (e & 1);
                        lt_split_store(ahi + t * 24 + s, alo + t * 24 + s, s <= t ? q[n][e] * pw[t - s] : 0.f);
                    }
            }
        } else {
            // decays before each token (for r) and after it (for k), channel by channel
            for (int x = tid; x < 2 * DP; x += nthr) {
                const int ch = x % DP;
                if (!OUT && x >= DP) break;
                // everything is read before anything is written, so that the loads overlap
                const bf16 *src = x < DP ? kk : rr;
                float raw16[16], w16[16];
#pragma unroll
                for (int t = 0; t < 16; t++) {
                    raw16[t] = to_f32(src[t * KE + ch]);
                    w16[t] = t < nt ? ww[t * DP + ch] : 1.f;
                }
                float p = 1.f;
                if (x < DP) {
#pragma unroll
                    for (int t = 15; t >= 0; t--) {
                        lt_split_store(khi + t * KE + ch, klo + t * KE + ch, raw16[t] * p);
                        p *= w16[t];
                    }
                    sD[ch] = p;
                    if (!OUT) sP[ch] *= p;
                } else {
#pragma unroll
                    for (int t = 0; t < 16; t++) {
                        if (MODE == LS_UPDATED) p *= w16[t];
                        lt_split_store(rhi + t * KE + ch, rlo + t * KE + ch, raw16[t] * p);
                        if (MODE != LS_UPDATED) p *= w16[t];
                    }
                }
            }
            if (OUT) {
                // eight lanes share a column s of A; lane q takes channels 4 q .. 4 q + 3, 4 (q + 8) .., ...; a warp's four
                // columns lie four apart
                constexpr int C4 = DP / 32;
                const int q = lane & 7;
                for (int s0 = warp; s0 < 4; s0 += NW) {
                    const int s = s0 + 4 * (lane >> 3);
                    float x[C4][4], b = 0.f;
                    auto row4 = [&](const bf16 *p, int i, float (&o)[4]) {
                        const uint2 w = *reinterpret_cast<const uint2 *>(p + 4 * (q + 8 * i));
                        o[0] = bf16_lo(w.x), o[1] = bf16_hi(w.x), o[2] = bf16_lo(w.y), o[3] = bf16_hi(w.y);
                    };
#pragma unroll
                    for (int i = 0; i < C4; i++) {
                        const int ch = 4 * (q + 8 * i);
                        float r4[4];
                        row4(kk + s * KE, i, x[i]);
                        row4(rr + s * KE, i, r4);
                        const float4 u4 = !a.u ? make_float4(1.f, 1.f, 1.f, 1.f) : ch < a.dim ? *reinterpret_cast<const float4 *>(a.u + h * a.dim + ch) : make_float4(0.f, 0.f, 0.f, 0.f);
                        b = fmaf(r4[0] * u4.x, x[i][0], b);
                        b = fmaf(r4[1] * u4.y, x[i][1], b);
                        b = fmaf(r4[2] * u4.z, x[i][2], b);
                        b = fmaf(r4[3] * u4.w, x[i][3], b);
                    }
                    float v[16];
#pragma unroll
                    for (int t = 0; t < 16; t++) {
                        v[t] = t == s ? b : 0.f;
                        if (t > s) {
#pragma unroll
                            for (int i = 0; i < C4; i++) {
                                float r4[4];
                                row4(rr + t * KE, i, r4);
                                const float4 w4 = *reinterpret_cast<const float4 *>(ww + t * DP + 4 * (q + 8 * i));
                                const float wv[4] = {w4.x, w4.y, w4.z, w4.w};
#pragma unroll
                                for (int e = 0; e < 4; e++) {
                                    if (MODE == LS_UPDATED) x[i][e] *= wv[e];
                                    v[t] = fmaf(r4[e], x[i][e], v[t]);
                                    if (MODE != LS_UPDATED) x[i][e] *= wv[e];
                                }
                            }
                        }
                    }
                    // sums over the eight lanes; lane q ends up with rows q and q + 8
                    float keep[2] = {0.f, 0.f};
#pragma unroll
                    for (int t = 0; t < 16; t++) {
                        v[t] += __shfl_xor_sync(0xffffffffu, v[t], 1);
                        v[t] += __shfl_xor_sync(0xffffffffu, v[t], 2);
                        v[t] += __shfl_xor_sync(0xffffffffu, v[t], 4);
                        if (q == (t & 7)) keep[t >> 3] = v[t];
                    }
#pragma unroll
                    for (int i = 0; i < 2; i++) lt_split_store(ahi + (q + 8 * i) * 24 + s, alo + (q + 8 * i) * 24 + s, keep[i]);
                }
            }
        }
        __syncthreads();
        // v^T fragments: (columns, tokens) from [token][column] rows
        uint32_t va[4];
        lt_ldmatrix_x4_trans(va, base + (uint32_t)(it & 1) * L.stage + L.v + (uint32_t)((mi >> 1) * 8 + mr) * L.vp + (uint32_t)(warp * 32 + (mi & 1) * 16));
        if (OUT) {
            float o[2][4] = {};
            const uint32_t rb = CONST_W ? base + (uint32_t)(it & 1) * L.stage : base + L.rhi;
#pragma unroll
            for (int ks = 0; ks < DT; ks++) {
                uint32_t sh[4], sl[4], r4[4];
                lt_split(S[2 * ks][0], S[2 * ks][1], sh[0], sl[0]);
                lt_split(S[2 * ks][2], S[2 * ks][3], sh[1], sl[1]);
                lt_split(S[2 * ks + 1][0], S[2 * ks + 1][1], sh[2], sl[2]);
                lt_split(S[2 * ks + 1][2], S[2 * ks + 1][3], sh[3], sl[3]);
                lt_ldmatrix_x4(r4, rb + b_plain + (uint32_t)ks * 32u);
                lt_mma(o[0], sh, r4[0], r4[1]);
                lt_mma(o[1], sh, r4[2], r4[3]);
                lt_mma(o[0], sl, r4[0], r4[1]);
                lt_mma(o[1], sl, r4[2], r4[3]);
                if (!CONST_W) {
                    lt_ldmatrix_x4(r4, base + L.rlo + b_plain + (uint32_t)ks * 32u);
                    lt_mma(o[0], sh, r4[0], r4[1]);
                    lt_mma(o[1], sh, r4[2], r4[3]);
                }
            }
            if (CONST_W) {
#pragma unroll
                for (int n = 0; n < 2; n++)
#pragma unroll
                    for (int e = 0; e < 4; e++) o[n][e] *= pw[n * 8 + 2 * tq + (e & 1) + 1];
            }
            uint32_t ab[4];
            const uint32_t aa = (uint32_t)((mi >> 1) * 8 + mr) * 48u + (uint32_t)(mi & 1) * 16u;
            lt_ldmatrix_x4(ab, base + L.ahi + aa);
            lt_mma(o[0], va, ab[0], ab[1]);
            lt_mma(o[1], va, ab[2], ab[3]);
            lt_ldmatrix_x4(ab, base + L.alo + aa);
            lt_mma(o[0], va, ab[0], ab[1]);
            lt_mma(o[1], va, ab[2], ab[3]);
#pragma unroll
            for (int n = 0; n < 2; n++)
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const int t = n * 8 + 2 * tq + (e & 1), j = jw + g + 8 * (e >> 1);
                    if (t < nt && j < a.vdim) a.o[((size_t)(t0 + t) * a.heads + h) * a.vdim + j] = o[n][e] * a.o_mul;
                }
        }
#pragma unroll
        for (int np = 0; np < DT; np++) {
            uint32_t kb[4];
            float d0[2], d1[2];
            if (CONST_W) {
                d0[0] = d0[1] = d1[0] = d1[1] = pw[nt];
            } else {
                const float2 x = *reinterpret_cast<const float2 *>(sD + np * 16 + 2 * tq), y = *reinterpret_cast<const float2 *>(sD + np * 16 + 8 + 2 * tq);
                d0[0] = x.x, d0[1] = x.y, d1[0] = y.x, d1[1] = y.y;
            }
#pragma unroll
            for (int e = 0; e < 4; e++) {
                S[2 * np][e] *= d0[e & 1];
                S[2 * np + 1][e] *= d1[e & 1];
            }
            lt_ldmatrix_x4_trans(kb, base + L.khi + b_trans + (uint32_t)np * 32u);
            lt_mma(S[2 * np], va, kb[0], kb[1]);
            lt_mma(S[2 * np + 1], va, kb[2], kb[3]);
            lt_ldmatrix_x4_trans(kb, base + L.klo + b_trans + (uint32_t)np * 32u);
            lt_mma(S[2 * np], va, kb[0], kb[1]);
            lt_mma(S[2 * np + 1], va, kb[2], kb[3]);
        }
        __syncthreads();   // this stage and the processed rows may be overwritten now
    }
    if (OUT) {
        if (c == a.n_chunks - 1) state_io(a.state, true);
    } else {
        state_io(a.starts + (size_t)c * cs, true);
        if (!CONST_W && blockIdx.z == 0)
            for (int ch = tid; ch < a.dim; ch += nthr) a.decays[((size_t)c * a.heads + h) * a.dim + ch] = sP[ch];
    }
}

// ---- few tokens: everything between the projections in one launch -------------------------------
// True for the one of n CTAs that arrives last at the counter (zero between launches); what the others wrote before is
// then visible to it through L2.
__device__ __forceinline__ bool last_of_head(int *counter, int n) {
    __shared__ int s_last;
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) {
        const int before = n > 1 ? atomicAdd(counter, 1) : 0;
        s_last = before == n - 1;
        if (n > 1 && s_last) *counter = 0;
        __threadfence();
    }
    __syncthreads();
    return s_last != 0;
}
// Head h of head_norm_gate_kernel for T tokens, f32, by one CTA; o [T][heads][vdim] is read through L2.
__device__ __forceinline__ void head_norm_gate_rows(const float *o, const float *g, const float *norm, float *act, int T, int heads, int h, int vdim, int norm_head,
                                                    int ldg, int lda, float eps, float mul) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    for (int t = warp; t < T; t += nw) {
        const float *x = o + ((size_t)t * heads + h) * vdim;
        float ss = 0.f;
        for (int i = lane; i < vdim; i += 32) {
            const float v = __ldcg(x + i);
            ss = fmaf(v, v, ss);
        }
        const float r = mul / sqrtf(warp_sum(ss) / (float)vdim + eps);
        const float *gt = g + (size_t)t * ldg + (size_t)h * vdim;
        float *at = act + (size_t)t * lda + (size_t)h * vdim;
        for (int i = lane; i < vdim; i += 32) at[i] = __ldcg(x + i) * r * (norm ? norm[(size_t)h * norm_head + i] : 1.0f) * silu_f32(gt[i]);
    }
}
struct LinearStepArgs {
    const float *r, *k, *v, *g;      // projections of the tokens, f32: [tokens][heads * dim] (v, g: heads * vdim), rows of ldr, ldv
    const float *z, *w0, *decay, *u; // low-rank decays: z [tokens][rank], w0 [heads * dim]; u [heads * dim] or null; retention: decay [heads]
    const bf16 *w2;                  // [heads * dim][rank]
    const float *norm;               // null: 1, else `norm_head` elements from one head's to the next
    Rotation rot;                    // of r and k (table null: none)
    const int *pos0;
    float k_mul, o_mul, out_mul, inv_tau, eps;   // o_mul before the norm, out_mul after the gate
    float *state, *o, *act;          // o: scratch [tokens][heads * vdim]; act: the output, rows of lda
    int *counters;                   // [heads], zero between launches
    int tokens, heads, dim, vdim, rank, mode, norm_head, ldr, ldv, lda;
};
__host__ inline size_t linear_step_smem(int tokens, int dim, int rank) {
    return sizeof(float) * ((size_t)tokens * (3 * dim + rank + 32 + 1) + 8 * 32);
}
// grid = (heads, ceil(vdim / 32)), 256 threads: lane = value column, warp w holds channels w, w + 8, ...
// (TI of them).  The CTA of a head that finishes last normalises and gates the head's outputs.
template <int TI>
RNB_GLOBAL void __launch_bounds__(256)
linear_state_step_kernel(const __grid_constant__ LinearStepArgs a) {
    extern __shared__ __align__(16) float st_smem[];
    pdl_launch_dependents();
    const int T = a.tokens, dim = a.dim, vdim = a.vdim, h = blockIdx.x, j0 = blockIdx.y * 32;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, j = j0 + lane;
    const bool live = j < vdim;
    float *sr = st_smem, *sk = sr + T * dim, *sw = sk + T * dim, *sz = sw + T * dim, *sv = sz + T * a.rank, *sb = sv + T * 32, *red = sb + T;
    // four lanes per channel of the decay product; the first 64 channels' weights are loaded ahead of the wait
    const int dch = tid >> 2, dl = tid & 3, seg = a.rank / 4;
    const bool dvec = !a.decay && a.rank % 32 == 0 && a.rank <= 128;
    uint4 dw[4];
    if (dvec && dch < dim)
#pragma unroll
        for (int i = 0; i < 4; i++)
            if (i * 8 < seg) dw[i] = ldg_nc_u4(a.w2 + ((size_t)h * dim + dch) * a.rank + dl * seg + i * 8);
    float *sp = a.state + (size_t)h * dim * vdim + j;
    if (vdim * 4 >= 128) {
        for (int ch = tid; ch < dim; ch += 256) asm volatile("prefetch.global.L2 [%0];" ::"l"(a.state + ((size_t)h * dim + ch) * vdim + j0));
    } else if (blockIdx.y == 0) {
        prefetch_l2(a.state + (size_t)h * dim * vdim, (size_t)dim * vdim * 4, tid, 256);
    }
    pdl_wait();
    float S[TI];
#pragma unroll
    for (int q = 0; q < TI; q++) {
        const int ch = warp + 8 * q;
        S[q] = live && ch < dim ? sp[(size_t)ch * vdim] : 0.f;
    }
    const int p0 = a.rot.table ? *a.pos0 : 0;
    for (int i = tid; i < T * dim; i += 256) {
        const int t = i / dim, ch = i % dim;
        const float *rr = a.r + (size_t)t * a.ldr + h * dim, *kk = a.k + (size_t)t * a.ldr + h * dim;
        sr[i] = rotated_element(a.rot, p0 + t, ch, [&](int e) { return rr[e]; });
        sk[i] = rotated_element(a.rot, p0 + t, ch, [&](int e) { return kk[e]; }) * a.k_mul;
        if (a.decay) sw[i] = a.decay[h];
    }
    for (int i = tid; i < T * 32; i += 256) {
        const int col = j0 + (i & 31);
        sv[i] = col < vdim ? a.v[(size_t)(i >> 5) * a.ldv + h * vdim + col] : 0.f;
    }
    for (int i = tid; i < T * a.rank; i += 256) sz[i] = a.mode == LS_BONUS ? tanhf(a.z[i]) : a.z[i];
    __syncthreads();
    const int dkind = a.mode == LS_UPDATED ? DECAY_SIGMOID_ROOT : DECAY_EXP;
    if (dvec) {
        for (int ch = dch; ch < (dim + 63) / 64 * 64; ch += 64) {
            if (ch != dch && ch < dim)
#pragma unroll
                for (int i = 0; i < 4; i++)
                    if (i * 8 < seg) dw[i] = ldg_nc_u4(a.w2 + ((size_t)h * dim + ch) * a.rank + dl * seg + i * 8);
            for (int t = 0; t < T; t++) {
                float s = 0.f;
                const float *z = sz + t * a.rank + dl * seg;
                if (ch < dim)
#pragma unroll
                    for (int i = 0; i < 4; i++)
                        if (i * 8 < seg) {
                            const uint32_t p[4] = {dw[i].x, dw[i].y, dw[i].z, dw[i].w};
#pragma unroll
                            for (int e = 0; e < 4; e++) {
                                s = fmaf(bf16_lo(p[e]), z[i * 8 + 2 * e], s);
                                s = fmaf(bf16_hi(p[e]), z[i * 8 + 2 * e + 1], s);
                            }
                        }
                s += __shfl_xor_sync(0xffffffffu, s, 1);
                s += __shfl_xor_sync(0xffffffffu, s, 2);
                if (dl == 0 && ch < dim) sw[t * dim + ch] = decay_of(dkind, s + a.w0[h * dim + ch], a.inv_tau);
            }
        }
    } else if (!a.decay) {
        for (int ch = warp; ch < dim; ch += 8) {
            const bf16 *w = a.w2 + ((size_t)h * dim + ch) * a.rank;
            for (int t = 0; t < T; t++) {
                float s = 0.f;
                for (int q = lane; q < a.rank; q += 32) s = fmaf(to_f32(w[q]), sz[t * a.rank + q], s);
                s = warp_sum(s);
                if (lane == 0) sw[t * dim + ch] = decay_of(dkind, s + a.w0[h * dim + ch], a.inv_tau);
            }
        }
    }
    for (int t = warp; t < T; t += 8) {
        float b = 0.f;
        for (int ch = lane; ch < dim; ch += 32) b = fmaf(sr[t * dim + ch] * (a.u ? a.u[h * dim + ch] : 1.f), sk[t * dim + ch], b);
        b = warp_sum(b);
        if (lane == 0) sb[t] = b;
    }
    __syncthreads();
    const float rs = a.decay ? a.decay[h] : 1.f;
    for (int t = 0; t < T; t++) {
        const float v = sv[t * 32 + lane];
        float acc = 0.f;
#pragma unroll
        for (int q = 0; q < TI; q++) {
            const int ch = warp + 8 * q;
            if (ch < dim) {
                acc = fmaf(a.mode == LS_UPDATED ? sr[t * dim + ch] * sw[t * dim + ch] : sr[t * dim + ch], S[q], acc);
                S[q] = fmaf(sw[t * dim + ch], S[q], sk[t * dim + ch] * v);
            }
        }
        red[warp * 32 + lane] = acc;
        __syncthreads();
        if (warp == 0) {
            float s = 0.f;
#pragma unroll
            for (int i = 0; i < 8; i++) s += red[i * 32 + lane];
            if (live) __stcg(a.o + ((size_t)t * a.heads + h) * vdim + j, fmaf(rs, s, sb[t] * v) * a.o_mul);
        }
        __syncthreads();
    }
#pragma unroll
    for (int q = 0; q < TI; q++) {
        const int ch = warp + 8 * q;
        if (live && ch < dim) sp[(size_t)ch * vdim] = S[q];
    }
    if (last_of_head(a.counters + h, gridDim.y)) head_norm_gate_rows(a.o, a.g, a.norm, a.act, T, a.heads, h, vdim, a.norm_head, a.ldv, a.lda, a.eps, a.out_mul);
}

}  // namespace rnb
