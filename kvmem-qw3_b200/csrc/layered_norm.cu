// Residual addition, the loop's additions and the RMS norm that follows, in one launch (layered models).
#include "layered.h"

namespace {

constexpr int LN_THREADS = 256;

// One CTA per row; the row lives in shared memory as fp32.
template <typename T>
__global__ void __launch_bounds__(LN_THREADS)
layer_norm_kernel(QbLayerNorm a) {
    QB_PDL_ENTER();
    extern __shared__ float row[];
    __shared__ float red[LN_THREADS / 32];
    const uint32_t m = blockIdx.x, n = a.n;
    const uint32_t src = a.row_map ? (uint32_t)a.row_map[m] : m;
    float *x = a.x + (size_t)src * n;
    if (a.tokens) {
        const uint32_t t = (uint32_t)a.tokens[m];
        const __nv_bfloat16 *e = a.embed + (size_t)(t < a.vocab ? t : 0) * n;
        float ss = 0.0f;
        for (uint32_t i = threadIdx.x; i < n; i += LN_THREADS) {
            const float v = __bfloat162float(e[i]);
            row[i] = v;
            ss += v * v;
        }
        const float inv = rsqrtf(qb_block_sum(ss, red, LN_THREADS / 32) / (float)n + a.eps);
        for (uint32_t i = threadIdx.x; i < n; i += LN_THREADS) row[i] = row[i] * inv * a.embed_w[i];
    } else {
        const size_t ps = (size_t)a.M * n;
        for (uint32_t i = threadIdx.x; i < n; i += LN_THREADS) {
            float v = x[i];
            if (a.S) v += qb_ldsum(a.parts, (size_t)m * n + i, a.S, ps);
            row[i] = v;
        }
    }
    float ss = 0.0f;
    for (uint32_t i = threadIdx.x; i < n; i += LN_THREADS) {       // a thread touches its own elements only
        float v = row[i];
        if (a.trace) a.trace[(size_t)m * n + i] = v;
        if (a.emb_store) a.emb_store[(size_t)m * n + i] = v;
        if (a.emb_add) v += a.emb_add[(size_t)m * n + i];
        if (a.step) v += a.step[i];
        if (!a.row_map) x[i] = v;
        row[i] = v;
        ss += v * v;
    }
    if (!a.w) return;
    const float inv = rsqrtf(qb_block_sum(ss, red, LN_THREADS / 32) / (float)n + a.eps);
    T *out = (T *)a.out.p + (size_t)m * a.out.ld;
    for (uint32_t i = threadIdx.x; i < n; i += LN_THREADS) out[i] = qb_cast<T>(row[i] * inv * a.w[i]);
}

}  // namespace

int qb_launch_layer_norm(qb_ctx *ctx, const QbLayerNorm &a) {
    const size_t smem = (size_t)a.n * sizeof(float);
    QB_REQUIRE(a.M > 0 && smem <= 200 * 1024, "layer norm: rows of %u elements", a.n);
    QB_REQUIRE(!a.w || (a.M <= a.out.cap && a.n <= a.out.ld), "layer norm: %u rows of %u elements exceed the output buffer", a.M, a.n);
    if (a.out.f32) {
        QB_CUDA(cudaFuncSetAttribute(layer_norm_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        QB_CUDA(qb_launch_pdl(ctx->stream, layer_norm_kernel<float>, dim3(a.M), dim3(LN_THREADS), smem, a));
    } else {
        QB_CUDA(cudaFuncSetAttribute(layer_norm_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        QB_CUDA(qb_launch_pdl(ctx->stream, layer_norm_kernel<__nv_bfloat16>, dim3(a.M), dim3(LN_THREADS), smem, a));
    }
    QB_LAUNCHED(ctx, "layer_norm_kernel");
    return QB_OK;
}
