// Residual addition, the loop's additions and the RMS norm that follows, in one launch (layered models).
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
template <int V> __device__ __forceinline__ float sq(const Vec<V> &a) {
    float s = 0.0f;
#pragma unroll
    for (int i = 0; i < V; ++i) s += a.v[i] * a.v[i];
    return s;
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
        float ss = 0.0f;
#pragma unroll
        for (int k = 0; k < NE; ++k) {
            const uint32_t i = (tid + k * LN_THREADS) * V;
            if (i < n) { row[k] = ld<V>(e + i); ss += sq(row[k]); }
        }
        const float inv = rsqrtf(qb_block_sum(ss, red, LN_THREADS / 32) / (float)n + a.eps);
#pragma unroll
        for (int k = 0; k < NE; ++k) {
            const uint32_t i = (tid + k * LN_THREADS) * V;
            if (i < n) {
                const Vec<V> w = ld<V>(a.embed_w + i);
#pragma unroll
                for (int j = 0; j < V; ++j) row[k].v[j] = row[k].v[j] * inv * w.v[j];
            }
        }
    } else {
        const size_t ps = (size_t)a.M * n;
#pragma unroll
        for (int k = 0; k < NE; ++k) {
            const uint32_t i = (tid + k * LN_THREADS) * V;
            if (i < n) {
                row[k] = ld<V>(x + i);
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
                    add(row[k], sum);
                }
            }
        }
    }
    float ss = 0.0f;
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
            ss += sq(row[k]);
        }
    }
    if (!a.w) return;
    const float inv = rsqrtf(qb_block_sum(ss, red, LN_THREADS / 32) / (float)n + a.eps);
    T *out = (T *)a.out.p + (size_t)m * a.out.ld;
#pragma unroll
    for (int k = 0; k < NE; ++k) {
        const uint32_t i = (tid + k * LN_THREADS) * V;
        if (i < n) {
            Vec<V> w = ld<V>(a.w + i);
#pragma unroll
            for (int j = 0; j < V; ++j) w.v[j] = row[k].v[j] * inv * w.v[j];
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
    QB_REQUIRE(!a.w || (a.M <= a.out.cap && a.n <= a.out.ld), "layer norm: %u rows of %u elements exceed the output buffer", a.M, a.n);
    if (a.n % 4 == 0) return a.out.f32 ? launch<float, 4>(ctx, a) : launch<__nv_bfloat16, 4>(ctx, a);
    return a.out.f32 ? launch<float, 1>(ctx, a) : launch<__nv_bfloat16, 1>(ctx, a);
}
