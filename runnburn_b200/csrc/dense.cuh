// Dense (bf16) weight matrices of the layered decoders: y[t][row] = sum_k W[row][k] * x[t][k].
//
//   dense_gemv_kernel       1..8 tokens, f32 activations: one warp per two rows, weights streamed by
//                           16-byte loads (the first ones issued before the dependency wait)
//   dense_gemm_kernel       many tokens, bf16 activations, tcgen05: 128 rows x 256 tokens per CTA
//   dense_gemm_simt_kernel  many tokens in true f32 (and bf16 activations whose rows are not
//                           16-byte aligned, which the tiled copies cannot describe)
//
// All accumulate in f32.  Matrices that go out together share a launch (jobs).  A job with w2 is a
// gate + up pair: the result is act(w x) * (w2 x), act the tanh form of gelu or silu.
#pragma once
#include <cuda_bf16.h>

#include "common.cuh"
#include "prefill_gemm.cuh"

namespace rnb {

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }
template <class T>
__device__ __forceinline__ T from_f32(float v);
template <>
__device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float gelu_tanh_f32(float z) {
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
// The same through 0.5 (1 + tanh a) = 1 / (1 + exp(-2 a)), for results that are rounded to bf16 next: the fast
// exponential's and division's errors (about 2^-21) disappear in that rounding.
__device__ __forceinline__ float gelu_tanh_fast(float z) {
    return __fdividef(z, 1.0f + __expf(-1.5957691216057308f * (z + 0.044715f * z * z * z)));
}
__device__ __forceinline__ float silu_f32(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float bf16_lo(uint32_t w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float bf16_hi(uint32_t w) { return __uint_as_float(w & 0xffff0000u); }

__device__ __forceinline__ float silu_fast(float z) { return __fdividef(z, 1.0f + __expf(-z)); }
constexpr int ACT_GELU_TANH = 0, ACT_SILU = 1;
__device__ __forceinline__ float gate_act(int act, float z) { return act == ACT_SILU ? silu_f32(z) : gelu_tanh_f32(z); }
__device__ __forceinline__ float gate_act_fast(int act, float z) { return act == ACT_SILU ? silu_fast(z) : gelu_tanh_fast(z); }

// A decay in (0, 1) from its projection x: exp(-exp(x)), or sigmoid(x)^inv_tau taken through the logarithm of the sigmoid
// (whose absolute error is what counts for the power).
constexpr int DECAY_EXP = 0, DECAY_SIGMOID_ROOT = 1;
__device__ __forceinline__ float decay_of(int kind, float x, float inv_tau) {
    return kind == DECAY_SIGMOID_ROOT ? expf((fminf(x, 0.f) - logf(1.0f + expf(-fabsf(x)))) * inv_tau) : expf(-expf(x));
}
// sigmoid(x)^inv_tau for tensor-core products, whose operands were rounded to bf16: the fast exponential and logarithm
// (absolute error of the logarithm 2^-21).
__device__ __forceinline__ float sigmoid_root_fast(float x, float inv_tau) {
    return __expf((fminf(x, 0.f) - __logf(1.0f + __expf(-fabsf(x)))) * inv_tau);
}

constexpr int DENSE_MAX_JOBS = 6;

// ---- few tokens ---------------------------------------------------------------------------------
struct DenseVecJob {
    const bf16 *w, *w2;   // [rows][cols]; w2: the up half of a gate + up pair
    const float *x;       // token t at x + t * ldx
    float *y;             // token t at y + t * ldy
    int rows, cols, ldx, ldy, cta0, vec, act;   // vec: rows of 16-byte aligned weights (cols % 8 == 0) and inputs
};
struct DenseVecJobs {
    DenseVecJob j[DENSE_MAX_JOBS];
    int n, ksplit;   // ksplit (1, 2, 4): warps that share a pair of rows, each taking every ksplit-th 1024 columns
};
constexpr int DV_WARPS = 4, DV_UNROLL = 4;

// ksplit warps own two output rows (or the gate and the up row of one output).  T = tokens, 1 .. 8.
template <int T>
RNB_GLOBAL void __launch_bounds__(DV_WARPS * 32)
dense_gemv_kernel(const __grid_constant__ DenseVecJobs jobs) {
    pdl_launch_dependents();
    int js = 0;
    for (int i = 1; i < jobs.n; i++)
        if ((int)blockIdx.x >= jobs.j[i].cta0) js = i;
    const DenseVecJob &job = jobs.j[js];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int ks = jobs.ksplit, part = warp & (ks - 1);
    const int unit = ((int)blockIdx.x - job.cta0) * (DV_WARPS / ks) + warp / ks;
    __shared__ float s_part[DV_WARPS][2][T];
    const bool pair = job.w2 != nullptr;
    const int r0 = pair ? unit : 2 * unit, rows = job.rows, cols = job.cols;
    const bool live = r0 < rows, two = pair || r0 + 1 < rows;
    const bf16 *w0 = job.w + (size_t)min(r0, rows - 1) * cols;
    const bf16 *w1 = pair ? job.w2 + (size_t)min(r0, rows - 1) * cols : job.w + (size_t)min(r0 + 1, rows - 1) * cols;
    float a0[T], a1[T];
#pragma unroll
    for (int t = 0; t < T; t++) a0[t] = a1[t] = 0.f;
    if (job.vec) {
        uint4 b0[DV_UNROLL], b1[DV_UNROLL];
        const uint4 z4 = make_uint4(0u, 0u, 0u, 0u);
        auto fetch = [&](int k0) {
#pragma unroll
            for (int u = 0; u < DV_UNROLL; u++) {
                const int k = k0 + u * 256 + lane * 8;
                b0[u] = k < cols ? ldg_nc_u4(w0 + k) : z4;
                b1[u] = k < cols ? ldg_nc_u4(w1 + k) : z4;
            }
        };
        const int step = 256 * DV_UNROLL * ks;
        fetch(part * 256 * DV_UNROLL);        // weights do not depend on the previous launch
        pdl_wait();
        for (int k0 = part * 256 * DV_UNROLL; k0 < cols; k0 += step) {
            uint4 c0[DV_UNROLL], c1[DV_UNROLL];
#pragma unroll
            for (int u = 0; u < DV_UNROLL; u++) c0[u] = b0[u], c1[u] = b1[u];
            if (k0 + step < cols) fetch(k0 + step);
#pragma unroll
            for (int u = 0; u < DV_UNROLL; u++) {
                const int k = k0 + u * 256 + lane * 8;
                if (k >= cols) continue;
                const uint32_t p[4] = {c0[u].x, c0[u].y, c0[u].z, c0[u].w}, q[4] = {c1[u].x, c1[u].y, c1[u].z, c1[u].w};
#pragma unroll
                for (int t = 0; t < T; t++) {
                    const float4 xa = *reinterpret_cast<const float4 *>(job.x + (size_t)t * job.ldx + k);
                    const float4 xb = *reinterpret_cast<const float4 *>(job.x + (size_t)t * job.ldx + k + 4);
                    const float xv[8] = {xa.x, xa.y, xa.z, xa.w, xb.x, xb.y, xb.z, xb.w};
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        a0[t] = fmaf(bf16_lo(p[e]), xv[2 * e], a0[t]);
                        a0[t] = fmaf(bf16_hi(p[e]), xv[2 * e + 1], a0[t]);
                        a1[t] = fmaf(bf16_lo(q[e]), xv[2 * e], a1[t]);
                        a1[t] = fmaf(bf16_hi(q[e]), xv[2 * e + 1], a1[t]);
                    }
                }
            }
        }
    } else {
        pdl_wait();
        for (int k = part * 32 + lane; k < cols; k += 32 * ks) {
            const float p = to_f32(w0[k]), q = to_f32(w1[k]);
#pragma unroll
            for (int t = 0; t < T; t++) {
                const float xv = job.x[(size_t)t * job.ldx + k];
                a0[t] = fmaf(p, xv, a0[t]);
                a1[t] = fmaf(q, xv, a1[t]);
            }
        }
    }
#pragma unroll
    for (int t = 0; t < T; t++) a0[t] = warp_sum(a0[t]), a1[t] = warp_sum(a1[t]);
    if (ks > 1) {
        if (lane == 0)
#pragma unroll
            for (int t = 0; t < T; t++) s_part[warp][0][t] = a0[t], s_part[warp][1][t] = a1[t];
        __syncthreads();
        if (lane == 0 && part == 0)
            for (int w = 1; w < ks; w++)
#pragma unroll
                for (int t = 0; t < T; t++) a0[t] += s_part[warp + w][0][t], a1[t] += s_part[warp + w][1][t];
    }
    if (lane == 0 && live && part == 0) {
#pragma unroll
        for (int t = 0; t < T; t++) {
            float *y = job.y + (size_t)t * job.ldy + r0;
            if (pair) {
                y[0] = gate_act(job.act, a0[t]) * a1[t];
            } else {
                y[0] = a0[t];
                if (two) y[1] = a1[t];
            }
        }
    }
}

// ---- many tokens, tcgen05 -----------------------------------------------------------------------
// One CTA: 128 weight rows (M operand, TMEM lane = row) x 256 tokens (N operand), f32 accumulators in
// 256 tensor-memory columns.  K advances 64 per stage; a stage is one copy of 256 tokens and two of 64
// weight rows (a gate + up pair takes its second half from the other matrix), both in the 128-byte
// swizzle the descriptors expect, zeros past either end.  Two stages of 48 KB let two CTAs share an SM:
// one's epilogue overlaps the other's matmul.  Warp 0 issues the copies, warp 1 the MMAs, warps 2-5
// read the accumulators back.  Every wait is bounded; after a timeout the error flag is set, the
// copies in flight are waited for and the tensor memory is freed.
// grid = (token tiles, row tiles of all jobs): CTAs that run together share weight rows, so a weight matrix
// larger than L2 still crosses DRAM once.
constexpr int DG_TOK = 256, DG_ROWS = 128, DG_K = 64, DG_STAGES = 2, DG_THREADS = 192;
constexpr uint32_t DG_X_BYTES = DG_TOK * 128, DG_W_BYTES = DG_ROWS * 128, DG_STAGE_BYTES = DG_X_BYTES + DG_W_BYTES;
constexpr size_t DG_SMEM = (size_t)DG_STAGES * DG_STAGE_BYTES + 1024;

struct DenseGemmJob {
    void *y;             // [seq][ld]
    const float *decay_bias;   // not null: y = decay_of(w x + bias[row])
    float inv_tau;
    int rows, cols, tile0, out_bf16, pair, ld, act, decay_kind;
};
struct DenseGemmJobs {
    DenseGemmJob j[DENSE_MAX_JOBS];
    int n, seq;
};
struct DenseMaps {   // per job: tokens, weights, second weights
    PgTensorMap x[DENSE_MAX_JOBS], w[DENSE_MAX_JOBS], w2[DENSE_MAX_JOBS];
};

template <class OT>
__device__ __forceinline__ void dg_store(void *y, size_t idx, float v) { reinterpret_cast<OT *>(y)[idx] = from_f32<OT>(v); }

RNB_GLOBAL void __launch_bounds__(DG_THREADS)
dense_gemm_kernel(const __grid_constant__ DenseGemmJobs jobs, const __grid_constant__ DenseMaps maps, int *__restrict__ err_flag) {
    extern __shared__ __align__(1024) uint8_t dg_smem_raw[];
    __shared__ __align__(8) uint64_t full[DG_STAGES], empty[DG_STAGES], done_bar;
    __shared__ uint32_t tmem_slot;
    __shared__ int s_failed;
    pdl_launch_dependents();
    uint8_t *smem = reinterpret_cast<uint8_t *>((reinterpret_cast<uintptr_t>(dg_smem_raw) + 1023) & ~(uintptr_t)1023);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    int js = 0;
    for (int i = 1; i < jobs.n; i++)
        if ((int)blockIdx.y >= jobs.j[i].tile0) js = i;
    const DenseGemmJob &job = jobs.j[js];
    const bool pair = job.pair != 0;
    const int rows = job.rows, seq = jobs.seq;
    const int n0 = ((int)blockIdx.y - job.tile0) * (pair ? DG_ROWS / 2 : DG_ROWS), m0 = blockIdx.x * DG_TOK;
    const int KT = (job.cols + DG_K - 1) / DG_K;
    if (tid == 0) {
        for (int s = 0; s < DG_STAGES; s++) {
            mbar_init(&full[s], 1);
            mbar_init(&empty[s], 1);
        }
        mbar_init(&done_bar, 1);
        mbar_fence_init();
        s_failed = 0;
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_slot)), "r"(256) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    pg_fence_before();
    __syncthreads();
    pg_fence_after();
    const uint32_t tmem = tmem_slot;
    pdl_wait();

    if (warp == 0) {
        if (lane == 0) {
            bool ok = true;
            int issued = 0;
            for (int kt = 0; kt < KT && ok; kt++) {
                const int s = kt % DG_STAGES;
                ok = mbar_wait_bounded(&empty[s], (uint32_t)(((kt / DG_STAGES) & 1) ^ 1));
                if (!ok) break;
                const uint32_t dst = smem_u32(smem + (uint32_t)s * DG_STAGE_BYTES);
                mbar_arrive_expect_tx(&full[s], DG_STAGE_BYTES);
                pg_tma_2d(dst, &maps.x[js], kt * DG_K, m0, &full[s]);
                pg_tma_2d(dst + DG_X_BYTES, &maps.w[js], kt * DG_K, n0, &full[s]);
                pg_tma_2d(dst + DG_X_BYTES + DG_W_BYTES / 2, pair ? &maps.w2[js] : &maps.w[js], kt * DG_K, pair ? n0 : n0 + DG_ROWS / 2, &full[s]);
                issued = kt + 1;
            }
            if (!ok) {
                // copies that were announced must land before the CTA may leave
                atomicExch(&s_failed, 1);
                for (int kt = max(0, issued - DG_STAGES); kt < issued; kt++) mbar_wait_bounded(&full[kt % DG_STAGES], (uint32_t)((kt / DG_STAGES) & 1));
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            bool ok = true;
            for (int kt = 0; kt < KT && ok; kt++) {
                const int s = kt % DG_STAGES;
                ok = mbar_wait_bounded(&full[s], (uint32_t)((kt / DG_STAGES) & 1));
                if (!ok) break;
                pg_fence_after();
                const uint32_t x_addr = smem_u32(smem + (uint32_t)s * DG_STAGE_BYTES), w_addr = x_addr + DG_X_BYTES;
#pragma unroll
                for (int k = 0; k < 4; k++)
                    pg_mma(tmem, pg_smem_desc(w_addr + (uint32_t)k * 32u), pg_smem_desc(x_addr + (uint32_t)k * 32u), (kt > 0 || k > 0) ? 1u : 0u);
                pg_commit(&empty[s]);
            }
            if (ok) pg_commit(&done_bar);
            else atomicExch(&s_failed, 1);
        }
    } else {
        const int q = warp & 3;   // tensor-memory lane quarter of this warp
        const bool fin = mbar_wait_bounded(&done_bar, 0u);
        if (!fin) atomicExch(&s_failed, 1);
        pg_fence_after();
        const int n_cc = min(DG_TOK, seq - m0 + 31) / 32;   // 32-token column groups that hold tokens
        if (pair) {
            // gate rows on lanes 0-63, the same rows of up on lanes 64-127: the four warps exchange them through
            // shared memory (the stages are free: every MMA has been committed) and each finishes 16 of the 32 tokens
            float *ex = reinterpret_cast<float *>(smem);
            const int qp = q & 1, t_lo = (q >> 1) * 16;
            const int row = n0 + qp * 32 + lane;
            for (int cc = 0; cc < n_cc; cc++) {
                float *buf = ex + (size_t)(cc & 1) * (4 * 32 * 33);
                float *mine = buf + (size_t)q * (32 * 33);
                const float *gs = buf + (size_t)qp * (32 * 33), *us = buf + (size_t)(qp + 2) * (32 * 33);
                uint32_t v[32];
                if (fin) pg_tmem_ld32(tmem + ((uint32_t)(q * 32) << 16) + (uint32_t)(cc * 32), v);
#pragma unroll
                for (int i = 0; i < 32; i++) mine[lane * 33 + i] = fin ? __uint_as_float(v[i]) : 0.f;
                asm volatile("bar.sync 1, 128;" ::: "memory");
                if (fin && row < rows) {
#pragma unroll
                    for (int i = 0; i < 16; i++) {
                        const int tok = m0 + cc * 32 + t_lo + i;
                        const float z = gs[lane * 33 + t_lo + i];
                        const float a = (job.out_bf16 ? gate_act_fast(job.act, z) : gate_act(job.act, z)) * us[lane * 33 + t_lo + i];
                        if (tok < seq) {
                            if (job.out_bf16) dg_store<bf16>(job.y, (size_t)tok * job.ld + row, a);
                            else dg_store<float>(job.y, (size_t)tok * job.ld + row, a);
                        }
                    }
                }
            }
        } else if (fin) {
            const int row = n0 + q * 32 + lane;
            for (int cc = 0; cc < n_cc; cc++) {
                uint32_t v[32];
                pg_tmem_ld32(tmem + ((uint32_t)(q * 32) << 16) + (uint32_t)(cc * 32), v);
                if (row < rows) {
                    if (job.decay_bias) {
                        const float b = job.decay_bias[row];
                        if (job.decay_kind == DECAY_SIGMOID_ROOT) {
#pragma unroll
                            for (int i = 0; i < 32; i++) v[i] = __float_as_uint(sigmoid_root_fast(__uint_as_float(v[i]) + b, job.inv_tau));
                        } else {
#pragma unroll
                            for (int i = 0; i < 32; i++) v[i] = __float_as_uint(expf(-expf(__uint_as_float(v[i]) + b)));
                        }
                    }
#pragma unroll
                    for (int i = 0; i < 32; i++) {
                        const int tok = m0 + cc * 32 + i;
                        if (tok < seq) {
                            if (job.out_bf16) dg_store<bf16>(job.y, (size_t)tok * job.ld + row, __uint_as_float(v[i]));
                            else dg_store<float>(job.y, (size_t)tok * job.ld + row, __uint_as_float(v[i]));
                        }
                    }
                }
            }
        }
    }
    pg_fence_before();
    __syncthreads();
    if (warp == 1) {
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(256) : "memory");
        if (lane == 0 && s_failed && err_flag) atomicExch(err_flag, DEV_ERR_GEMM_TIMEOUT);
    }
}

// ---- many tokens, f32 arithmetic on the CUDA cores ----------------------------------------------
struct DenseSimtJob {
    const bf16 *w, *w2;
    const void *x;       // [seq][ldx] of XT
    void *y;             // [seq][ld]
    int rows, cols, tile0, out_bf16, ldx, ld, act;
};
struct DenseSimtJobs {
    DenseSimtJob j[DENSE_MAX_JOBS];
    int n, seq;
};
constexpr int DS_TILE = 64, DS_K = 16;
// grid = (row tiles of all jobs, token tiles), 256 threads, a 4 x 4 block of outputs per thread
template <class XT>
RNB_GLOBAL void __launch_bounds__(256)
dense_gemm_simt_kernel(const __grid_constant__ DenseSimtJobs jobs) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float xs[DS_K][DS_TILE + 4], ws[DS_K][DS_TILE + 4], us[DS_K][DS_TILE + 4];
    int js = 0;
    for (int i = 1; i < jobs.n; i++)
        if ((int)blockIdx.x >= jobs.j[i].tile0) js = i;
    const DenseSimtJob &job = jobs.j[js];
    const bool pair = job.w2 != nullptr;
    const XT *x = reinterpret_cast<const XT *>(job.x);
    const int n0 = ((int)blockIdx.x - job.tile0) * DS_TILE, m0 = blockIdx.y * DS_TILE;
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    float a[4][4] = {}, b[4][4] = {};
    for (int k0 = 0; k0 < job.cols; k0 += DS_K) {
        for (int i = tid; i < DS_TILE * DS_K; i += 256) {
            const int k = i & (DS_K - 1), r = i / DS_K;
            const bool kin = k0 + k < job.cols;
            xs[k][r] = kin && m0 + r < jobs.seq ? to_f32(x[(size_t)(m0 + r) * job.ldx + k0 + k]) : 0.f;
            const bool win = kin && n0 + r < job.rows;
            ws[k][r] = win ? to_f32(job.w[(size_t)(n0 + r) * job.cols + k0 + k]) : 0.f;
            if (pair) us[k][r] = win ? to_f32(job.w2[(size_t)(n0 + r) * job.cols + k0 + k]) : 0.f;
        }
        __syncthreads();
        float c[4][4] = {}, d[4][4] = {};   // sums of sums: rounding grows with the depth of one tile and the number of tiles
#pragma unroll
        for (int k = 0; k < DS_K; k++) {
            const float4 xv = *reinterpret_cast<const float4 *>(&xs[k][ty * 4]), wv = *reinterpret_cast<const float4 *>(&ws[k][tx * 4]);
            const float xr[4] = {xv.x, xv.y, xv.z, xv.w}, wr[4] = {wv.x, wv.y, wv.z, wv.w};
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) c[i][j] = fmaf(xr[i], wr[j], c[i][j]);
            if (pair) {
                const float4 uv = *reinterpret_cast<const float4 *>(&us[k][tx * 4]);
                const float ur[4] = {uv.x, uv.y, uv.z, uv.w};
#pragma unroll
                for (int i = 0; i < 4; i++)
#pragma unroll
                    for (int j = 0; j < 4; j++) d[i][j] = fmaf(xr[i], ur[j], d[i][j]);
            }
        }
#pragma unroll
        for (int i = 0; i < 4; i++)
#pragma unroll
            for (int j = 0; j < 4; j++) a[i][j] += c[i][j], b[i][j] += d[i][j];
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int tok = m0 + ty * 4 + i, row = n0 + tx * 4 + j;
            if (tok >= jobs.seq || row >= job.rows) continue;
            const float v = pair ? gate_act(job.act, a[i][j]) * b[i][j] : a[i][j];
            if (job.out_bf16) dg_store<bf16>(job.y, (size_t)tok * job.ld + row, v);
            else dg_store<float>(job.y, (size_t)tok * job.ld + row, v);
        }
}

}  // namespace rnb
