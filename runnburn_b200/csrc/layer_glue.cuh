// Row-wise kernels of the layered decoders: embedding, residual + norms (+ token shift), rotations,
// head norm + gate.  Everything here computes in f32; activations leave as HT (f32, or bf16 where
// the next matmul runs on tcgen05).
#pragma once
#include "dense.cuh"

namespace rnb {

// Sum over the CTA (any multiple of 32 threads up to 1024), returned to every thread.
__device__ __forceinline__ float block_sum(float v, float *red) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    v = warp_sum(v);
    __syncthreads();   // the previous use of red is over
    if (lane == 0) red[warp] = v;
    __syncthreads();
    v = lane < nw ? red[lane] : 0.f;
    return warp_sum(v);
}

// Weights do not depend on the launch before: asking for them ahead of the dependency wait hides their DRAM latency.
__device__ __forceinline__ void prefetch_l2(const void *p, size_t bytes, int tid, int nthreads) {
    if (!p) return;
    for (size_t i = (size_t)tid * 128; i < bytes; i += (size_t)nthreads * 128) asm volatile("prefetch.global.L2 [%0];" ::"l"((const char *)p + i));
}

// grid = tokens.  x and (when kept for later passes) emb: [tokens][width] f32
RNB_GLOBAL void __launch_bounds__(256)
dense_embed_kernel(const bf16 *__restrict__ table, const uint32_t *__restrict__ token, int width, float scale, float *__restrict__ x, float *__restrict__ emb) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t row = (size_t)token[blockIdx.x] * width, o = (size_t)blockIdx.x * width;
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        const float v = to_f32(table[row + i]) * scale;
        x[o + i] = v;
        if (emb) emb[o + i] = v;
    }
}

// The end of one sublayer and the start of the next in one pass over the residual rows:
//   x <- x + mult * (y / rms(y)) * (1 + wb) + emb     (y, emb: may be null; wb null: x + mult * y + emb)
//   h <- (x / rms(x)) * (1 + wn)                      (wn null: stop at x)
//   or, with `center`, the layer norm  h <- (x - mean) / sqrt(mean (x - mean)^2 + eps) * wn + bn
// With mu [n_mix][width] the output is n_mix token-shifted mixes  h + (h' - h) * mu_s  instead, stream s
// at h + s * tokens * width; h' is the previous token's h, which the CTA recomputes for the row before its
// first (from x_in, so x_out must be another buffer when there are several CTAs) or takes from shift_in
// for the step's first token.  The last token's h goes to shift_out.
// grid = ceil(tokens / rows_per_cta); dynamic shared memory (mu ? 2 : 1) * width floats.
struct ResidualNormArgs {
    const float *x_in, *y, *wb, *emb, *wn, *bn, *mu, *shift_in;
    float *x_out, *shift_out;
    void *h;
    float mult, eps;
    int width, tokens, rows_per_cta, n_mix, center;
};
template <class HT, int V>   // V: elements per access (4 when width % 4 == 0, else 1)
RNB_GLOBAL void __launch_bounds__(1024)
residual_norm_kernel(const __grid_constant__ ResidualNormArgs a) {
    extern __shared__ __align__(16) float rn_smem[];
    __shared__ float red[32];
    pdl_launch_dependents();
    if (gridDim.x == 1) {
        prefetch_l2(a.wb, (size_t)a.width * 4, threadIdx.x, blockDim.x);
        prefetch_l2(a.wn, (size_t)a.width * 4, threadIdx.x, blockDim.x);
        prefetch_l2(a.bn, (size_t)a.width * 4, threadIdx.x, blockDim.x);
        prefetch_l2(a.mu, (size_t)a.width * 4 * a.n_mix, threadIdx.x, blockDim.x);
    }
    pdl_wait();
    struct alignas(4 * V) Vec { float v[V]; };
    struct alignas(sizeof(HT) * V) HVec { HT v[V]; };
    const int D = a.width, step = blockDim.x * V;
    float *cur = rn_smem, *prev = rn_smem + D;
    HT *h = reinterpret_cast<HT *>(a.h);
    const int t0 = blockIdx.x * a.rows_per_cta, t1 = min(t0 + a.rows_per_cta, a.tokens);
    for (int t = (a.mu && t0 > 0) ? t0 - 1 : t0; t < t1; t++) {
        const size_t row = (size_t)t * D;
        const bool mine = t >= t0;
        float ry = 0.f;
        if (a.y && a.wb) {
            float ss = 0.f;
            for (int i = threadIdx.x * V; i < D; i += step) {
                const Vec y = *reinterpret_cast<const Vec *>(a.y + row + i);
#pragma unroll
                for (int e = 0; e < V; e++) ss = fmaf(y.v[e], y.v[e], ss);
            }
            ry = 1.0f / sqrtf(block_sum(ss, red) / (float)D + a.eps);
        }
        float ss = 0.f;
        for (int i = threadIdx.x * V; i < D; i += step) {
            Vec x = *reinterpret_cast<const Vec *>(a.x_in + row + i);
            if (a.y) {
                const Vec y = *reinterpret_cast<const Vec *>(a.y + row + i);
                if (a.wb) {
                    const Vec w = *reinterpret_cast<const Vec *>(a.wb + i);
#pragma unroll
                    for (int e = 0; e < V; e++) x.v[e] += a.mult * (y.v[e] * ry * (1.0f + w.v[e]));
                } else {
#pragma unroll
                    for (int e = 0; e < V; e++) x.v[e] = fmaf(a.mult, y.v[e], x.v[e]);
                }
            }
            if (a.emb) {
                const Vec z = *reinterpret_cast<const Vec *>(a.emb + row + i);
#pragma unroll
                for (int e = 0; e < V; e++) x.v[e] += z.v[e];
            }
            if (mine && (a.y || a.emb || a.x_out != a.x_in)) *reinterpret_cast<Vec *>(a.x_out + row + i) = x;
            *reinterpret_cast<Vec *>(cur + i) = x;
#pragma unroll
            for (int e = 0; e < V; e++) ss = a.center ? ss + x.v[e] : fmaf(x.v[e], x.v[e], ss);
        }
        if (!a.wn) continue;
        float mean = 0.f;
        if (a.center) {
            mean = block_sum(ss, red) / (float)D;
            ss = 0.f;
            for (int i = threadIdx.x * V; i < D; i += step) {
                const Vec c = *reinterpret_cast<const Vec *>(cur + i);   // this thread's own elements
#pragma unroll
                for (int e = 0; e < V; e++) ss = fmaf(c.v[e] - mean, c.v[e] - mean, ss);
            }
        }
        const float rx = 1.0f / sqrtf(block_sum(ss, red) / (float)D + a.eps);
        for (int i = threadIdx.x * V; i < D; i += step) {
            Vec c = *reinterpret_cast<const Vec *>(cur + i);   // this thread's own elements
            const Vec w = *reinterpret_cast<const Vec *>(a.wn + i);
#pragma unroll
            for (int e = 0; e < V; e++) c.v[e] = a.center ? (c.v[e] - mean) * rx * w.v[e] : c.v[e] * rx * (1.0f + w.v[e]);
            if (a.bn) {
                const Vec b = *reinterpret_cast<const Vec *>(a.bn + i);
#pragma unroll
                for (int e = 0; e < V; e++) c.v[e] += b.v[e];
            }
            if (a.mu) {
                Vec p;
                if (t == 0) p = *reinterpret_cast<const Vec *>(a.shift_in + i);
                else p = *reinterpret_cast<const Vec *>(prev + i);
                *reinterpret_cast<Vec *>(prev + i) = c;
                if (t == a.tokens - 1) *reinterpret_cast<Vec *>(a.shift_out + i) = c;
                if (!mine) continue;
                for (int s = 0; s < a.n_mix; s++) {
                    const Vec mu = *reinterpret_cast<const Vec *>(a.mu + (size_t)s * D + i);
                    HVec o;
#pragma unroll
                    for (int e = 0; e < V; e++) o.v[e] = from_f32<HT>(c.v[e] + (p.v[e] - c.v[e]) * mu.v[e]);
                    *reinterpret_cast<HVec *>(h + (size_t)s * a.tokens * D + row + i) = o;
                }
            } else {
                HVec o;
#pragma unroll
                for (int e = 0; e < V; e++) o.v[e] = from_f32<HT>(c.v[e]);
                *reinterpret_cast<HVec *>(h + row + i) = o;
            }
        }
    }
}

// Norm of selected residual rows (the final norm of the positions whose logits are wanted): with b the
// layer norm of weight w and bias b, without it the root-mean-square norm of weight 1 + w.
// rows null: row blockIdx.x itself.  grid = rows, dynamic shared memory none.
template <class HT>
RNB_GLOBAL void __launch_bounds__(512)
norm_rows_kernel(const float *__restrict__ x, const int *__restrict__ rows, const float *__restrict__ w, const float *__restrict__ b, float eps, int width,
                 HT *__restrict__ h) {
    __shared__ float red[32];
    pdl_launch_dependents();
    pdl_wait();
    const float *xs = x + (size_t)(rows ? rows[blockIdx.x] : (int)blockIdx.x) * width;
    float mean = 0.f, ss = 0.f;
    if (b) {
        for (int i = threadIdx.x; i < width; i += blockDim.x) mean += xs[i];
        mean = block_sum(mean, red) / (float)width;
    }
    for (int i = threadIdx.x; i < width; i += blockDim.x) ss = fmaf(xs[i] - mean, xs[i] - mean, ss);
    const float r = 1.0f / sqrtf(block_sum(ss, red) / (float)width + eps);
    HT *hs = h + (size_t)blockIdx.x * width;
    for (int i = threadIdx.x; i < width; i += blockDim.x) hs[i] = from_f32<HT>(b ? (xs[i] - mean) * r * w[i] + b[i] : xs[i] * r * (1.0f + w[i]));
}

// ---- rotary positions ---------------------------------------------------------------------------
// table [position][dims / 2] of (cos, sin), any scaling of the two included.  Pair i of a vector is
// (2i, 2i + 1) when interleaved, else (i, i + dims / 2).
struct Rotation {
    const float2 *table;
    int dims, interleaved;
};
__device__ __forceinline__ void rotation_pair(const Rotation &r, int i, int &a, int &b) {
    a = r.interleaved ? 2 * i : i;
    b = r.interleaved ? 2 * i + 1 : i + r.dims / 2;
}
// Element e of the rotated vector; src(e) reads the unrotated one.
template <class Src>
__device__ __forceinline__ float rotated_element(const Rotation &r, int pos, int e, Src src) {
    if (!r.table || e >= r.dims) return src(e);
    const int half = r.dims / 2;
    const int i = r.interleaved ? e >> 1 : (e < half ? e : e - half);
    const bool second = r.interleaved ? (e & 1) : e >= half;
    int a, b;
    rotation_pair(r, i, a, b);
    const float2 cs = r.table[(size_t)pos * half + i];
    const float u = src(a), v = src(b);
    return second ? fmaf(v, cs.x, u * cs.y) : fmaf(u, cs.x, -(v * cs.y));
}
// In place over [tokens][heads][hd] rows: the vector of a head starts `off` elements into it; afterwards
// the whole head is multiplied by `mul`.  grid = (tokens, 1 or 2 buffers), position = *pos0 + token.
struct RotateArgs {
    void *x[2];
    float mul[2];
    int heads, hd, off;
    Rotation rot;
    const int *pos0;
};
template <class AT>
RNB_GLOBAL void __launch_bounds__(256)
rotate_heads_kernel(const __grid_constant__ RotateArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const int pos = *a.pos0 + (int)blockIdx.x, half = a.rot.dims / 2, rest = a.hd - a.rot.dims;
    AT *x = reinterpret_cast<AT *>(a.x[blockIdx.y]) + (size_t)blockIdx.x * a.heads * a.hd;
    const float mul = a.mul[blockIdx.y];
    for (int i = threadIdx.x; i < a.heads * half; i += blockDim.x) {
        AT *v = x + (size_t)(i / half) * a.hd + a.off;
        int p, q;
        rotation_pair(a.rot, i % half, p, q);
        const float2 cs = a.rot.table[(size_t)pos * half + i % half];
        const float u = to_f32(v[p]), w = to_f32(v[q]);
        v[p] = from_f32<AT>(fmaf(u, cs.x, -(w * cs.y)) * mul);
        v[q] = from_f32<AT>(fmaf(w, cs.x, u * cs.y) * mul);
    }
    if (mul != 1.0f && rest > 0)
        for (int i = threadIdx.x; i < a.heads * rest; i += blockDim.x) {
            const int e = i % rest;   // the elements around the rotated part: [0, off) and [off + dims, hd)
            AT *v = x + (size_t)(i / rest) * a.hd + (e < a.off ? e : e + a.rot.dims);
            *v = from_f32<AT>(to_f32(*v) * mul);
        }
}

// act = (o / rms(o over the head)) * w * silu(g) * mul; w null: 1, else `w_head` elements from one head's to the
// next (0: shared by the heads).  `lanes` (a power of two up to 32) per (token, head), V elements per
// access (4 when vdim and the row strides are multiples of 4, else 1).
struct HeadNormGateArgs {
    const float *o, *w;      // [tokens][heads][vdim]
    const void *g;           // token t's rows at g + t * ldg, act + t * lda
    void *act;
    size_t units;            // tokens * heads
    float eps, mul;
    int heads, vdim, lanes, w_head, ldg, lda;
};
template <class HT, int V>
RNB_GLOBAL void __launch_bounds__(256)
head_norm_gate_kernel(const __grid_constant__ HeadNormGateArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    struct alignas(4 * V) Vec { float v[V]; };
    struct alignas(sizeof(HT) * V) HVec { HT v[V]; };
    const int lanes = a.lanes, vdim = a.vdim;
    const size_t unit = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) / lanes;
    const int l = threadIdx.x & (lanes - 1);
    const bool in = unit < a.units;
    const size_t u = in ? unit : 0, t = u / a.heads;
    const int h = (int)(u % a.heads);
    const float *o = a.o + u * vdim, *w = a.w ? a.w + (size_t)h * a.w_head : nullptr;
    float ss = 0.f;
    for (int j = l * V; j < vdim; j += lanes * V) {
        const Vec x = *reinterpret_cast<const Vec *>(o + j);
#pragma unroll
        for (int e = 0; e < V; e++) ss = fmaf(x.v[e], x.v[e], ss);
    }
    for (int d = 1; d < lanes; d <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, d);
    const float r = a.mul / sqrtf(ss / (float)vdim + a.eps);
    if (!in) return;
    const HT *g = reinterpret_cast<const HT *>(a.g) + t * a.ldg + (size_t)h * vdim;
    HT *act = reinterpret_cast<HT *>(a.act) + t * a.lda + (size_t)h * vdim;
    for (int j = l * V; j < vdim; j += lanes * V) {
        const Vec x = *reinterpret_cast<const Vec *>(o + j);
        const HVec y = *reinterpret_cast<const HVec *>(g + j);
        HVec out;
#pragma unroll
        for (int e = 0; e < V; e++) out.v[e] = from_f32<HT>(x.v[e] * r * (w ? w[j + e] : 1.0f) * silu_f32(to_f32(y.v[e])));
        *reinterpret_cast<HVec *>(act + j) = out;
    }
}

}  // namespace rnb
