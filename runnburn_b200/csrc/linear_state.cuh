// Linear recurrences with a matrix state per head (RWKV-style time mixing, retention), all in f32:
//   o_t = rs * S^T r_t + (sum_i r_t[i] u[i] k_t[i]) v_t,      S <- diag(w_t) S + k_t v_t^T
// Time mixing: w_t per key channel, u the bonus of the current token, rs = 1.  Retention, whose output
// reads the updated state S_t = decay S + k v^T: w_t = decay of the head, u = 1, rs = decay.
// State [heads][dim][vdim] f32.
//
//   linear_state_step_kernel    1..8 tokens, one launch: rotations or decays, recurrence, head norm, gate
//   linear_state_chunk_kernel   many tokens: the sequence is cut into chunks that run at the same time.
//       OUT = false: every chunk but the last accumulates its own contribution from a zero state;
//       linear_state_scan_kernel turns these into the state at the start of every chunk;
//       OUT = true: every chunk runs again from its start state and writes its outputs.
//     Decays enter as products of w, never as ratios of products: nothing can overflow.
#pragma once
#include "layer_glue.cuh"

namespace rnb {

struct LinearChunkArgs {
    const void *r, *k, *v;     // [tokens][heads][dim], same, [tokens][heads][vdim] (AT)
    const float *w;            // [tokens][heads][dim]; null: decay[head]
    const float *decay, *u;    // [heads]; [heads][dim], null: 1
    float *state, *o;          // [heads][dim][vdim]; [tokens][heads][vdim]
    float *starts, *decays;    // [chunks][heads][dim][vdim]; [chunks][heads][dim]
    int tokens, heads, dim, vdim, chunk, n_chunks;
    int G, JG;                 // lanes along dim (16 channels each), groups of 4 value columns per CTA
};
constexpr int LS_TI = 16, LS_TS = 16;   // channels per thread; tokens staged at a time
__host__ __device__ inline size_t linear_chunk_smem(int G, int JG) { return sizeof(float) * ((size_t)LS_TS * (3 * LS_TI * G + 4 * JG) + LS_TS); }

// grid = (chunks, heads, column blocks); G * JG threads rounded up to a warp.
// Thread (jg, g): value columns 4 jg .. + 3, channels 4 (q G + g) .. + 3 for q = 0..3.
template <class AT, bool OUT, bool CONST_W>
RNB_GLOBAL void __launch_bounds__(256)
linear_state_chunk_kernel(const __grid_constant__ LinearChunkArgs a) {
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
            const size_t at = ((size_t)(t0 + t) * a.heads + h) * a.dim + ch;
            if (OUT) sr[i] = in ? to_f32(rp[at]) : 0.f;
            sk[i] = in ? to_f32(kp[at]) : 0.f;
            if (!CONST_W) sw[i] = in ? a.w[at] : 0.f;
        }
        for (int i = tid; i < nt * VB; i += blockDim.x) {
            const int t = i / VB, col = j0 + i % VB;
            sv[i] = col < a.vdim ? to_f32(vp[((size_t)(t0 + t) * a.heads + h) * a.vdim + col]) : 0.f;
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
                        if (OUT) acc[e] = fmaf(rr[i], S[4 * q + i][e], acc[e]);
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
                        if (j + e < a.vdim) o[e] = fmaf(rs, acc[e], sb[t] * vv[e]);
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

// starts[c] <- the state at the start of chunk c, from the chunks' own contributions.  One thread per state element.
RNB_GLOBAL void __launch_bounds__(256)
linear_state_scan_kernel(const float *__restrict__ state, float *__restrict__ starts, const float *__restrict__ decays, const float *__restrict__ decay,
                         int heads, int dim, int vdim, int chunk, int n_chunks) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t n = (size_t)heads * dim * vdim, i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    const size_t row = i / vdim;
    float S = state[i];
    const float p0 = decays ? 0.f : powf(decay[row / dim], (float)chunk);
#pragma unroll 4
    for (int c = 0; c < n_chunks - 1; c++) {
        const float add = starts[(size_t)c * n + i], p = decays ? decays[(size_t)c * heads * dim + row] : p0;
        starts[(size_t)c * n + i] = S;
        S = fmaf(p, S, add);
    }
    starts[(size_t)(n_chunks - 1) * n + i] = S;
}

// Decays of time mixing: out[t][c] = exp(-exp(sum_j w2[c][j] tanh(z[t][j]) + w0[c])).
// grid = (ceil(channels / 128), ceil(tokens / 16)), 128 threads; dynamic shared memory 16 * rank floats.
RNB_GLOBAL void __launch_bounds__(128)
decay_rows_kernel(const float *__restrict__ z, const bf16 *__restrict__ w2, const float *__restrict__ w0, int tokens, int rank, int channels,
                  float *__restrict__ out) {
    extern __shared__ __align__(16) float dr_smem[];   // [rank][16]
    pdl_launch_dependents();
    pdl_wait();
    const int t0 = blockIdx.y * 16;
    for (int i = threadIdx.x; i < rank * 16; i += blockDim.x) {
        const int t = i / rank, j = i % rank;
        dr_smem[j * 16 + t] = t0 + t < tokens ? tanhf(z[(size_t)(t0 + t) * rank + j]) : 0.f;
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
        if (t0 + t < tokens) out[(size_t)(t0 + t) * channels + c] = expf(-expf(acc[t] + b));
}

// ---- few tokens: everything between the projections in one launch -------------------------------
struct LinearStepArgs {
    const float *r, *k, *v, *g;      // projections of the tokens, f32: [tokens][heads * dim] (v, g: heads * vdim)
    const float *z, *w0, *decay, *u; // time mixing: z [tokens][rank], w0 and u [heads * dim]; retention: decay [heads]
    const bf16 *w2;                  // [heads * dim][rank]
    const float *norm;               // [heads * vdim] or null
    Rotation rot;                    // of r and k (table null: none)
    const int *pos0;
    float k_mul, eps;
    float *state, *o, *act;          // o: scratch [tokens][heads * vdim]; act: the output
    int *counters;                   // [heads], zero between launches
    int tokens, heads, dim, vdim, rank;
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
    __shared__ int s_last;
    pdl_launch_dependents();
    pdl_wait();
    const int T = a.tokens, dim = a.dim, vdim = a.vdim, h = blockIdx.x, j0 = blockIdx.y * 32;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, j = j0 + lane;
    const bool live = j < vdim;
    float *sr = st_smem, *sk = sr + T * dim, *sw = sk + T * dim, *sz = sw + T * dim, *sv = sz + T * a.rank, *sb = sv + T * 32, *red = sb + T;
    float S[TI];
    float *sp = a.state + (size_t)h * dim * vdim + j;
#pragma unroll
    for (int q = 0; q < TI; q++) {
        const int ch = warp + 8 * q;
        S[q] = live && ch < dim ? sp[(size_t)ch * vdim] : 0.f;
    }
    const int p0 = a.rot.table ? *a.pos0 : 0;
    for (int i = tid; i < T * dim; i += 256) {
        const int t = i / dim, ch = i % dim;
        const float *rr = a.r + ((size_t)t * a.heads + h) * dim, *kk = a.k + ((size_t)t * a.heads + h) * dim;
        sr[i] = rotated_element(a.rot, p0 + t, ch, [&](int e) { return rr[e]; });
        sk[i] = rotated_element(a.rot, p0 + t, ch, [&](int e) { return kk[e]; }) * a.k_mul;
        if (a.decay) sw[i] = a.decay[h];
    }
    for (int i = tid; i < T * 32; i += 256) {
        const int col = j0 + (i & 31);
        sv[i] = col < vdim ? a.v[((size_t)(i >> 5) * a.heads + h) * vdim + col] : 0.f;
    }
    for (int i = tid; i < T * a.rank; i += 256) sz[i] = tanhf(a.z[i]);
    __syncthreads();
    if (!a.decay) {
        for (int ch = warp; ch < dim; ch += 8) {
            const bf16 *w = a.w2 + ((size_t)h * dim + ch) * a.rank;
            for (int t = 0; t < T; t++) {
                float s = 0.f;
                for (int q = lane; q < a.rank; q += 32) s = fmaf(to_f32(w[q]), sz[t * a.rank + q], s);
                s = warp_sum(s);
                if (lane == 0) sw[t * dim + ch] = expf(-expf(s + a.w0[h * dim + ch]));
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
                acc = fmaf(sr[t * dim + ch], S[q], acc);
                S[q] = fmaf(sw[t * dim + ch], S[q], sk[t * dim + ch] * v);
            }
        }
        red[warp * 32 + lane] = acc;
        __syncthreads();
        if (warp == 0) {
            float s = 0.f;
#pragma unroll
            for (int i = 0; i < 8; i++) s += red[i * 32 + lane];
            if (live) __stcg(a.o + ((size_t)t * a.heads + h) * vdim + j, fmaf(rs, s, sb[t] * v));
        }
        __syncthreads();
    }
#pragma unroll
    for (int q = 0; q < TI; q++) {
        const int ch = warp + 8 * q;
        if (live && ch < dim) sp[(size_t)ch * vdim] = S[q];
    }
    __threadfence();
    __syncthreads();
    if (tid == 0) {
        const int n = gridDim.y, before = n > 1 ? atomicAdd(a.counters + h, 1) : 0;
        s_last = before == n - 1;
        if (n > 1 && s_last) a.counters[h] = 0;
        __threadfence();
    }
    __syncthreads();
    if (!s_last) return;
    for (int t = warp; t < T; t += 8) {
        const size_t at = ((size_t)t * a.heads + h) * vdim;
        float ss = 0.f;
        for (int i = lane; i < vdim; i += 32) {
            const float v = __ldcg(a.o + at + i);
            ss = fmaf(v, v, ss);
        }
        const float r = 1.0f / sqrtf(warp_sum(ss) / (float)vdim + a.eps);
        for (int i = lane; i < vdim; i += 32)
            a.act[at + i] = __ldcg(a.o + at + i) * r * (a.norm ? a.norm[h * vdim + i] : 1.0f) * silu_f32(a.g[at + i]);
    }
}

}  // namespace rnb
