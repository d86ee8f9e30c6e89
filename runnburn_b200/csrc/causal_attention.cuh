// Causal softmax attention of a prompt's queries on tensor cores, bf16 operands, f32 scores and weights.
// A key may consist of a piece per key/value head and one that all heads share (latent attention's rotated part);
// query heads may share key/value heads; a window may bound how far back a query sees; keys and values may
// live in a ring (position p in row p % ring).  The output may be gated, one sigmoid per head.
#pragma once
#include "layer_glue.cuh"
#include "mma_bf16.cuh"

#include <limits.h>

namespace rnb {

constexpr int CA_ROWS = 128, CA_KEYS = 64, CA_THREADS = 256;
__host__ __device__ inline int ca_pad16(int n) { return (n + 15) & ~15; }
// columns of the value tile that the kernel is instantiated for: 32, 64, 128, 256 (0: too wide)
__host__ inline int causal_attention_vcols(int vdim) { return vdim <= 32 ? 32 : vdim <= 64 ? 64 : vdim <= 128 ? 128 : vdim <= 256 ? 256 : 0; }
__host__ inline size_t causal_attention_smem(int key_dim, int vdim) {
    return 2 * ((size_t)(CA_ROWS + 2 * CA_KEYS) * (ca_pad16(key_dim) + 8) + (size_t)2 * CA_KEYS * (causal_attention_vcols(vdim) + 8));
}
struct CausalAttentionArgs {
    const bf16 *q;                 // token t, head h: q + t * ldq + h * (dim + dim2)
    const bf16 *k, *k2, *v;        // row r: k + r * ldk + (h / group) * dim, k2 + r * ldk2 (dim2 elements), v + r * ldv + (h / group) * vdim
    bf16 *act;                     // [tokens][lda]
    const float *gate;             // null or [tokens][ldg]: the output of head h times sigmoid(gate[t][h])
    const int *pos0;
    size_t ldq, ldk, ldk2, ldv;
    float scale, out_mul;
    int tokens, heads, group, dim, dim2, vdim, ring, window, lda, ldg;   // window 0: everything before
    int vec;                       // every row piece is 16-byte aligned and a multiple of 8 elements
};
// grid = (ceil(tokens / 128), heads), 256 threads; warp w owns queries 16w .. 16w + 15 of the CTA's 128.
// Keys come in tiles of 64, double-buffered; the weights enter the value product as bf16 hi + lo parts.
// DVJ: 8-column tiles of the value dimension (vdim <= 8 DVJ).
template <int DVJ>
RNB_GLOBAL void __launch_bounds__(CA_THREADS, 1)
causal_attention_kernel(const __grid_constant__ CausalAttentionArgs a) {
    extern __shared__ __align__(128) uint8_t ca_smem[];
    pdl_launch_dependents();
    pdl_wait();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y;
    const int hk = h / a.group, dk = a.dim + a.dim2, dkp = ca_pad16(dk), KS = dkp / 16;
    constexpr int DVP = 8 * DVJ;
    const uint32_t kpitch = (uint32_t)(dkp + 8) * 2, vpitch = (uint32_t)(DVP + 8) * 2;
    bf16 *qs = reinterpret_cast<bf16 *>(ca_smem);
    bf16 *ks = qs + (size_t)CA_ROWS * (dkp + 8), *vs = ks + (size_t)2 * CA_KEYS * (dkp + 8);
    const uint32_t q_base = smem_u32(qs), k_base = smem_u32(ks), v_base = smem_u32(vs);
    const int i0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * CA_ROWS;   // long rows first
    const int pos0 = *a.pos0, kv_len = pos0 + a.tokens;
    const int n_keys = min(kv_len, pos0 + i0 + CA_ROWS), n_tiles = (n_keys + CA_KEYS - 1) / CA_KEYS;
    const int window = a.window > 0 ? a.window : INT_MAX;
    const int t_first = a.window > 0 ? max(0, pos0 + i0 - a.window + 1) / CA_KEYS : 0;
    const bf16 zero = from_f32<bf16>(0.f);
    // queries, and zeros in the padding columns of every buffer (the copies below never touch those)
    for (int i = tid; i < CA_ROWS * (dkp + 8); i += CA_THREADS) {
        const int r = i / (dkp + 8), c = i % (dkp + 8);
        qs[i] = c < dk && i0 + r < a.tokens ? a.q[(size_t)(i0 + r) * a.ldq + (size_t)h * dk + c] : zero;
    }
    if (dkp > dk)
        for (int i = tid; i < 2 * CA_KEYS * (dkp - dk); i += CA_THREADS) ks[(size_t)(i / (dkp - dk)) * (dkp + 8) + dk + i % (dkp - dk)] = zero;
    if (DVP > a.vdim)
        for (int i = tid; i < 2 * CA_KEYS * (DVP - a.vdim); i += CA_THREADS) vs[(size_t)(i / (DVP - a.vdim)) * (DVP + 8) + a.vdim + i % (DVP - a.vdim)] = zero;
    auto load_tile = [&](int t) {
        const int st = t & 1, key0 = t * CA_KEYS;
        if (a.vec) {
            // four threads walk along a key's rows
            const int r = tid >> 2, q0 = tid & 3, key = key0 + r, kk = min(key, kv_len - 1) % a.ring;
            const uint32_t nbytes = key < kv_len ? 16u : 0u;
            auto row = [&](uint32_t dst, const bf16 *src, int chunks) {
                for (int c = q0; c < chunks; c += 4)
                    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst + (uint32_t)c * 16u), "l"(src + c * 8), "r"(nbytes) : "memory");
            };
            const uint32_t kdst = k_base + (uint32_t)(st * CA_KEYS + r) * kpitch;
            row(kdst, a.k + (size_t)kk * a.ldk + (size_t)hk * a.dim, a.dim / 8);
            if (a.dim2) row(kdst + (uint32_t)a.dim * 2u, a.k2 + (size_t)kk * a.ldk2, a.dim2 / 8);
            row(v_base + (uint32_t)(st * CA_KEYS + r) * vpitch, a.v + (size_t)kk * a.ldv + (size_t)hk * a.vdim, a.vdim / 8);
        } else {
            const int per = dk + a.vdim;
            for (int i = tid; i < CA_KEYS * per; i += CA_THREADS) {
                const int r = i / per, c = i % per;
                const bool in = key0 + r < kv_len;
                const int key = (key0 + r) % a.ring;
                if (c < dk)
                    ks[(size_t)(st * CA_KEYS + r) * (dkp + 8) + c] =
                        !in ? zero : c < a.dim ? a.k[(size_t)key * a.ldk + (size_t)hk * a.dim + c] : a.k2[(size_t)key * a.ldk2 + c - a.dim];
                else
                    vs[(size_t)(st * CA_KEYS + r) * (DVP + 8) + c - dk] = in ? a.v[(size_t)key * a.ldv + (size_t)hk * a.vdim + c - dk] : zero;
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load_tile(t_first);
    const int g = lane >> 2, tq = lane & 3, mi = lane >> 3, mr = lane & 7;
    int qi[2], pos[2];
    bool live[2];
#pragma unroll
    for (int e = 0; e < 2; e++) {
        qi[e] = i0 + warp * 16 + g + 8 * e;
        live[e] = qi[e] < a.tokens;
        pos[e] = live[e] ? pos0 + qi[e] : kv_len - 1;   // rows past the end see what the last one sees and are never stored
    }
    float o[DVJ][4], m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
#pragma unroll
    for (int j = 0; j < DVJ; j++) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
    const float sl2 = a.scale * 1.4426950408889634f;
    // A fragments: matrices (rows 0-7, k 0-7), (rows 8-15, k 0-7), (rows 0-7, k 8-15), (rows 8-15, k 8-15)
    const uint32_t q_addr = q_base + (uint32_t)(warp * 16 + (mi & 1) * 8 + mr) * kpitch + (uint32_t)(mi >> 1) * 16u;
    for (int t = t_first; t < n_tiles; t++) {
        if (t + 1 < n_tiles) {
            load_tile(t + 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const uint32_t k_st = k_base + (uint32_t)(t & 1) * CA_KEYS * kpitch, v_st = v_base + (uint32_t)(t & 1) * CA_KEYS * vpitch;
        float s[8][4];
#pragma unroll
        for (int j = 0; j < 8; j++) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
        // B fragments of two key tiles per ldmatrix: (keys 0-7, k 0-7), (keys 0-7, k 8-15), (keys 8-15, k 0-7), (keys 8-15, k 8-15)
        const uint32_t kb = k_st + (uint32_t)((mi >> 1) * 8 + mr) * kpitch + (uint32_t)(mi & 1) * 16u;
#pragma unroll 4
        for (int kk = 0; kk < KS; kk++) {
            uint32_t af[4];
            lt_ldmatrix_x4(af, q_addr + (uint32_t)kk * 32u);
#pragma unroll
            for (int jp = 0; jp < 4; jp++) {
                uint32_t b[4];
                lt_ldmatrix_x4(b, kb + (uint32_t)(jp * 16) * kpitch + (uint32_t)kk * 32u);
                lt_mma(s[2 * jp], af, b[0], b[1]);
                lt_mma(s[2 * jp + 1], af, b[2], b[3]);
            }
        }
        const int key0 = t * CA_KEYS + 2 * tq;
        const bool need_mask = t * CA_KEYS + CA_KEYS - 1 > min(pos[0], pos[1]) || max(pos[0], pos[1]) - t * CA_KEYS >= window;
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int j = 0; j < 8; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                float x = s[j][e] * sl2;
                if (need_mask) {
                    const int back = pos[e >> 1] - (key0 + j * 8 + (e & 1));
                    if (back < 0 || back >= window) x = -INFINITY;
                }
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
            lt_split(p0, p1, ph[j >> 1][2 * (j & 1)], pl[j >> 1][2 * (j & 1)]);
            lt_split(p2, p3, ph[j >> 1][2 * (j & 1) + 1], pl[j >> 1][2 * (j & 1) + 1]);
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
                lt_ldmatrix_x4_trans(b, vb + (uint32_t)jp * 32u);
                lt_mma(o[2 * jp], ph[kk], b[0], b[1]);
                lt_mma(o[2 * jp], pl[kk], b[0], b[1]);
                lt_mma(o[2 * jp + 1], ph[kk], b[2], b[3]);
                lt_mma(o[2 * jp + 1], pl[kk], b[2], b[3]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int e = 0; e < 2; e++) {
        if (!live[e]) continue;
        float inv = a.out_mul / l_run[e];
        if (a.gate) inv /= 1.0f + expf(-a.gate[(size_t)qi[e] * a.ldg + h]);
        bf16 *dst = a.act + (size_t)qi[e] * a.lda + (size_t)h * a.vdim;
#pragma unroll
        for (int j = 0; j < DVJ; j++)
#pragma unroll
            for (int x = 0; x < 2; x++)
                if (8 * j + 2 * tq + x < a.vdim) dst[8 * j + 2 * tq + x] = from_f32<bf16>(o[j][2 * e + x] * inv);
    }
}

}  // namespace rnb
