// The residual stream between two sublayers in one launch (layered models): the sublayer's result -- plain, or normalised and
// weighted first -- joins the stream, then the loop's additions, then the norm of what follows (or its plain cast).
#include "layered.h"

namespace {

constexpr int LN_THREADS = 512;

// V consecutive elements of a row at a time: V = 4 where the rows allow 16-byte accesses, else 1.
template <int V> struct Vec { float v[V]; };
template <int V> __device__ __forceinline__ Vec<V> ld(const float *p) {
    Vec<V> r;
    if constexpr (V == 4) { const float4 f = *reinterpret_cast<const float4 *>(p); r.v[0] = f.x; r.v[1] = f.y; r.v[2] = f.z; r.v[3] = f.w; }
    else r.v[0] = *p;
    return r;
}
template <int V> __device__ __forceinline__ void st(float *p, const Vec<V> &r) {
    if constexpr (V == 4) *reinterpret_cast<float4 *>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else *p = r.v[0];
}
template <int V> __device__ __forceinline__ Vec<V> ld(const __nv_bfloat16 *p) {
    Vec<V> r;
#pragma unroll
    for (int i = 0; i < V; ++i) r.v[i] = __bfloat162float(p[i]);
    return r;
}
template <int V> __device__ __forceinline__ void st(__nv_bfloat16 *p, const Vec<V> &r) {
    if constexpr (V == 4) {
        __nv_bfloat162 b[2] = {__floats2bfloat162_rn(r.v[0], r.v[1]), __floats2bfloat162_rn(r.v[2], r.v[3])};
        *reinterpret_cast<uint2 *>(p) = *reinterpret_cast<const uint2 *>(b);
    } else *p = __float2bfloat16(r.v[0]);
}
template <int V> __device__ __forceinline__ void add(Vec<V> &a, const Vec<V> &b) {
#pragma unroll
    for (int i = 0; i < V; ++i) a.v[i] += b.v[i];
}
template <int V> __device__ __forceinline__ float sum(const Vec<V> &a) {
    float s = 0.0f;
#pragma unroll
    for (int i = 0; i < V; ++i) s += a.v[i];
    return s;
}
// squares of the deviations from a mean (0: plain squares)
template <int V> __device__ __forceinline__ float sq(const Vec<V> &a, float mean) {
    float s = 0.0f;
#pragma unroll
    for (int i = 0; i < V; ++i) { const float d = a.v[i] - mean; s += d * d; }
    return s;
}

// Mean (0 for an RMS norm) and 1 / root of the mean square of a row whose pieces a block's threads hold.
struct Moments { float mean, inv; };
template <int V, int NE>
__device__ __forceinline__ Moments moments(const Vec<V> (&row)[NE], const QbLayerNorm &a, float *red) {
    Moments r{0.0f, 1.0f};
    if (a.center) {
        float t = 0.0f;
#pragma unroll
        for (int k = 0; k < NE; ++k)
            if ((threadIdx.x + k * LN_THREADS) * V < a.n) t += sum(row[k]);
        r.mean = qb_block_sum(t, red, LN_THREADS / 32) / (float)a.n;
    }
    float ss = 0.0f;
#pragma unroll
    for (int k = 0; k < NE; ++k)
        if ((threadIdx.x + k * LN_THREADS) * V < a.n) ss += sq(row[k], r.mean);
    r.inv = rsqrtf(qb_block_sum(ss, red, LN_THREADS / 32) / (float)a.n + a.eps);
    return r;
}

// One CTA per row; a thread keeps its NE pieces of the row in registers.
template <typename T, int V, int NE>
__global__ void __launch_bounds__(LN_THREADS)
layer_norm_kernel(QbLayerNorm a) {
    QB_PDL_ENTER();
    __shared__ float red[LN_THREADS / 32];
    const uint32_t m = blockIdx.x, n = a.n, tid = threadIdx.x;
    uint32_t src = a.row_map ? (uint32_t)a.row_map[m] : m;
    if (a.row_map && src >= a.x_rows) {                                  // recorded, and row 0 read instead
        if (tid == 0) atomicExch(a.err_flag, 6001);
        src = 0;
    }
    float *x = a.x + (size_t)src * n;
    Vec<V> row[NE];
    if (a.tokens) {
        const uint32_t t = (uint32_t)a.tokens[m];
        const __nv_bfloat16 *e = a.embed + (size_t)(t < a.vocab ? t : 0) * n;
#pragma unroll
        for (int k = 0; k < NE; ++k) {
            const uint32_t i = (tid + k * LN_THREADS) * V;
            if (i < n) {
                row[k] = ld<V>(e + i);
#pragma unroll
                for (int j = 0; j < V; ++j) row[k].v[j] *= a.embed_scale;
            }
        }
        if (a.embed_w) {
            const Moments mo = moments<V, NE>(row, a, red);
#pragma unroll
            for (int k = 0; k < NE; ++k) {
                const uint32_t i = (tid + k * LN_THREADS) * V;
                if (i < n) {
                    const Vec<V> w = ld<V>(a.embed_w + i);
#pragma unroll
                    for (int j = 0; j < V; ++j) row[k].v[j] = (row[k].v[j] - mo.mean) * mo.inv * w.v[j];
                }
            }
        }
    } else {
        const size_t ps = (size_t)a.M * n;
        Vec<V> res[NE];
        float scale = 1.0f;
        if (a.row_ss) {                                           // the norm that the mixer left out of its rows
            float t = 0.0f;
            for (uint32_t i = 0; i < a.ss_n; ++i) t += a.row_ss[(size_t)m * a.ss_n + i];
            scale = rsqrtf(t / (float)a.ss_len + a.eps);
        }
#pragma unroll
        for (int k = 0; k < NE; ++k) {
            const uint32_t i = (tid + k * LN_THREADS) * V;
            if (i < n) {
                res[k] = ld<V>(x + i);
                if (a.S) {
                    const float *p = a.parts + (size_t)m * n + i;
                    Vec<V> sum = ld<V>(p);
                    if (a.S > 1) {                                // up to 8 segments, all loads in flight
                        Vec<V> q[7];
#pragma unroll
                        for (uint32_t s = 1; s < 8; ++s)
                            if (s < a.S) q[s - 1] = ld<V>(p + s * ps);
#pragma unroll
                        for (uint32_t s = 1; s < 8; ++s)
                            if (s < a.S) add(sum, q[s - 1]);
                    }
                    row[k] = sum;
#pragma unroll
                    for (int j = 0; j < V; ++j) row[k].v[j] *= scale;
                }
            }
        }
        if (a.post_w) {
            const Moments mo = moments<V, NE>(row, a, red);
#pragma unroll
            for (int k = 0; k < NE; ++k) {
                const uint32_t i = (tid + k * LN_THREADS) * V;
                if (i < n) {
                    const Vec<V> w = ld<V>(a.post_w + i);
#pragma unroll
                    for (int j = 0; j < V; ++j) row[k].v[j] = (row[k].v[j] - mo.mean) * mo.inv * w.v[j];
                }
            }
        }
#pragma unroll
        for (int k = 0; k < NE; ++k) {
            if ((tid + k * LN_THREADS) * V >= n) continue;
            if (a.S) add(row[k], res[k]);
            else row[k] = res[k];
        }
    }
#pragma unroll
    for (int k = 0; k < NE; ++k) {
        const uint32_t i = (tid + k * LN_THREADS) * V;
        if (i < n) {
            const size_t at = (size_t)m * n + i;
            if (a.trace) st<V>(a.trace + at, row[k]);
            if (a.emb_store) st<V>(a.emb_store + at, row[k]);
            if (a.emb_add) add(row[k], ld<V>(a.emb_add + at));
            if (a.step) add(row[k], ld<V>(a.step + i));
            if (!a.row_map) st<V>(x + i, row[k]);
        }
    }
    T *out = (T *)a.out.p + (size_t)m * a.out.ld;
    if (!a.w) {
#pragma unroll
        for (int k = 0; k < NE; ++k) {
            const uint32_t i = (tid + k * LN_THREADS) * V;
            if (i < n) st<V>(out + i, row[k]);
        }
        return;
    }
    const Moments mo = moments<V, NE>(row, a, red);
#pragma unroll
    for (int k = 0; k < NE; ++k) {
        const uint32_t i = (tid + k * LN_THREADS) * V;
        if (i < n) {
            Vec<V> w = ld<V>(a.w + i);
#pragma unroll
            for (int j = 0; j < V; ++j) w.v[j] = (row[k].v[j] - mo.mean) * mo.inv * w.v[j];
            st<V>(out + i, w);
        }
    }
}

template <typename T, int V>
int launch(qb_ctx *ctx, const QbLayerNorm &a) {
    const uint32_t ne = (a.n + LN_THREADS * V - 1) / (LN_THREADS * V);
    QB_REQUIRE(ne <= 16, "layer norm: rows of %u elements", a.n);
    const dim3 grid(a.M), block(LN_THREADS);
    if (ne <= 1) QB_CUDA(qb_launch_pdl(ctx->stream, layer_norm_kernel<T, V, 1>, grid, block, (size_t)0, a));
    else if (ne <= 2) QB_CUDA(qb_launch_pdl(ctx->stream, layer_norm_kernel<T, V, 2>, grid, block, (size_t)0, a));
    else if (ne <= 4) QB_CUDA(qb_launch_pdl(ctx->stream, layer_norm_kernel<T, V, 4>, grid, block, (size_t)0, a));
    else QB_CUDA(qb_launch_pdl(ctx->stream, layer_norm_kernel<T, V, 16>, grid, block, (size_t)0, a));
    QB_LAUNCHED(ctx, "layer_norm_kernel");
    return QB_OK;
}

}  // namespace

int qb_launch_layer_norm(qb_ctx *ctx, const QbLayerNorm &args) {
    QbLayerNorm a = args;
    a.err_flag = ctx->err_flag_dev;
    QB_REQUIRE(a.M > 0, "layer norm: no rows");
    QB_REQUIRE(a.out.p && a.M <= a.out.cap && a.n <= a.out.ld, "layer norm: %u rows of %u elements exceed the output buffer", a.M, a.n);
    if (a.n % 4 == 0) return a.out.f32 ? launch<float, 4>(ctx, a) : launch<__nv_bfloat16, 4>(ctx, a);
    return a.out.f32 ? launch<float, 1>(ctx, a) : launch<__nv_bfloat16, 1>(ctx, a);
}
