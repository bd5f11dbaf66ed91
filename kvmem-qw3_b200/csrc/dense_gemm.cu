// Products with dense bfloat16 weights (the layered models): y = x W^T with fp32 accumulation.
//
// bfloat16 activations: tcgen05.mma kind::f16 (bf16 x bf16 -> fp32 in tensor memory), "swap-AB": the 128 weight rows of a
// CTA's tile are the MMA's M dimension, 16 .. 256 activation rows its N dimension, so that one kernel serves a single
// decode row and a prompt chunk.  Weights arrive as 16 KB records already in the swizzled operand order (one bulk copy per
// stage), activations by tensor-map TMA (128-byte swizzle, rows and columns outside the matrix read as zero).  Warp 0 is
// the producer, warp 1 issues the MMAs, the others drain the accumulator, which is double-buffered in tensor memory: the
// next unit's products run while a unit is written out.  The launch is a programmatic dependent one; the first weight
// stages are requested before the CTA waits for the kernel that produces the activations.  Every wait is bounded: when one
// runs out, the CTA raises the context's error flag, lets its copies land, frees its tensor memory and returns.
//
// fp32 activations: a plain fp32 FMA kernel (weights widened exactly).
#include "dense_gemm.h"
#include "tc_common.cuh"

#include <mutex>

namespace {
using namespace qbtc;

enum Epi { EPI_PARTS = 0, EPI_BF16 = 1, EPI_SWIGLU = 2 };

template <int NT>
struct DgCfg {
    static constexpr int CTAS = NT <= 32 ? 2 : 1;                     // resident CTAs per SM
    static constexpr int B_BYTES = NT * 128;
    static constexpr int STAGE = (int)QB_DREC_BYTES + B_BYTES;
    static constexpr int BAR_BYTES = 1024;
    static constexpr int FIT = (232448 / CTAS - BAR_BYTES - 2048) / STAGE;
    static constexpr int NST = FIT > 8 ? 8 : FIT;
    static constexpr int TOTAL = STAGE * NST + BAR_BYTES + 1024;      // + slack to align the base to 1024
    static constexpr int EPI_WARPS = NT >= 128 ? 8 : 4;
    static constexpr int THREADS = 64 + 32 * EPI_WARPS;
    static constexpr int NC = NT / (EPI_WARPS / 4);                   // accumulator columns per epilogue thread
    static constexpr uint32_t TMEM_COLS = 2 * NT;                     // two accumulators; a power of two >= 32
};

// Unit u of a launch: activation tile fastest (consecutive CTAs share a weight tile in L2), then K segment, then row tile.
template <int NT, int EPI>
__global__ void __launch_bounds__(DgCfg<NT>::THREADS, DgCfg<NT>::CTAS)
dense_gemm_kernel(const uint8_t *__restrict__ rec, const __grid_constant__ CUtensorMap map_x, uint32_t kc, uint32_t N, uint32_t M,
                  float *__restrict__ parts, __nv_bfloat16 *__restrict__ out, uint32_t ldo, uint32_t F, uint32_t S, uint32_t m_tiles, uint32_t units,
                  int *err_flag) {
    using C = DgCfg<NT>;
    constexpr uint32_t NST = C::NST;
    extern __shared__ uint8_t smem_raw[];
    uint8_t *smem = reinterpret_cast<uint8_t *>(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    uint8_t *bar_mem = smem + (size_t)C::STAGE * NST;
    // barriers: full[NST], empty[NST], acc_full[2], acc_empty[2]
    const uint32_t bar_full = smem_u32(bar_mem), bar_empty = bar_full + 8 * NST, bar_tfull = bar_empty + 8 * NST, bar_tempty = bar_tfull + 16;
    uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(bar_mem + 8 * (2 * NST + 4));
    volatile int *abort_flag = reinterpret_cast<volatile int *>(tmem_slot + 1);
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

    if (threadIdx.x == 0) {
        for (uint32_t i = 0; i < NST; ++i) { mbar_init(bar_full + 8 * i, 1); mbar_init(bar_empty + 8 * i, 1); }
        for (uint32_t i = 0; i < 2; ++i) { mbar_init(bar_tfull + 8 * i, 1); mbar_init(bar_tempty + 8 * i, C::EPI_WARPS); }
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(C::TMEM_COLS) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");

    auto decode = [&](uint32_t u, uint32_t &tile, uint32_t &seg, uint32_t &m0, uint32_t &c_begin, uint32_t &n_it) {
        m0 = (u % m_tiles) * NT;
        const uint32_t rest = u / m_tiles;
        seg = rest % S;
        tile = rest / S;
        c_begin = tc_seg_begin(seg, S, kc);
        n_it = tc_seg_begin(seg + 1, S, kc) - c_begin;
    };

    if (warp == 0) {
        if (lane == 0) {
            struct Cursor { uint32_t u, it, n_it, tile, m0, c_begin; bool valid; };
            auto start = [&](uint32_t u) {
                Cursor c; c.u = u; c.it = 0; c.valid = u < units; c.n_it = 0; c.tile = c.m0 = c.c_begin = 0;
                if (c.valid) { uint32_t seg; decode(u, c.tile, seg, c.m0, c.c_begin, c.n_it); }
                return c;
            };
            auto next = [&](Cursor &c) { if (++c.it >= c.n_it) c = start(c.u + gridDim.x); };
            auto load_w = [&](const Cursor &c, uint32_t st) {
                const uint32_t full = bar_full + 8 * st;
                mbar_expect_tx(full, C::STAGE);
                bulk_load(smem_u32(smem + (size_t)st * C::STAGE), rec + ((size_t)c.tile * kc + c.c_begin + c.it) * QB_DREC_BYTES, QB_DREC_BYTES, full);
            };
            auto load_x = [&](const Cursor &c, uint32_t st) {
                tma_load_2d(smem_u32(smem + (size_t)st * C::STAGE) + QB_DREC_BYTES, &map_x, (int)((c.c_begin + c.it) * 64), (int)c.m0, bar_full + 8 * st);
            };
            Cursor head = start(blockIdx.x), c = head;
            uint32_t npre = 0;
            for (; npre < NST && c.valid; ++npre, next(c)) load_w(c, npre);
            asm volatile("griddepcontrol.wait;" ::: "memory");
            c = head;
            for (uint32_t g = 0; g < npre; ++g, next(c)) load_x(c, g);
            for (uint32_t git = npre; c.valid; ++git, next(c)) {
                const uint32_t st = git % NST, ph = (git / NST) & 1;
                if (!mbar_wait(bar_empty + 8 * st, ph ^ 1, abort_flag)) break;
                load_w(c, st);
                load_x(c, st);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            // instruction descriptor: D fp32, A = B = bf16, both K-major, N = NT, M = 128
            constexpr uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(NT >> 3) << 17) | ((128u >> 4) << 24);
            uint32_t git = 0, j = 0;
            bool ok = true;
            for (uint32_t u = blockIdx.x; u < units && ok; u += gridDim.x, ++j) {
                uint32_t tile, seg, m0, c_begin, n_it;
                decode(u, tile, seg, m0, c_begin, n_it);
                const uint32_t ab = j & 1, aph = (j >> 1) & 1;
                if (!mbar_wait(bar_tempty + 8 * ab, aph ^ 1, abort_flag)) break;
                tc_fence_after();
                for (uint32_t it = 0; it < n_it; ++it, ++git) {
                    const uint32_t st = git % NST, ph = (git / NST) & 1;
                    if (!mbar_wait(bar_full + 8 * st, ph, abort_flag)) { ok = false; break; }
                    tc_fence_after();
                    const uint32_t a_addr = smem_u32(smem + (size_t)st * C::STAGE), b_addr = a_addr + QB_DREC_BYTES;
#pragma unroll
                    for (int ks = 0; ks < 4; ++ks)
                        tc_mma_f16(tmem_base + ab * NT, smem_desc_sw128(a_addr + ks * 32), smem_desc_sw128(b_addr + ks * 32), idesc,
                                    (it > 0 || ks > 0) ? 1u : 0u);
                    tc_commit(bar_empty + 8 * st);
                }
                if (ok) tc_commit(bar_tfull + 8 * ab);
            }
        }
    } else {
        const uint32_t quarter = warp & 3;                                // TMEM lanes [32 * quarter, +32)
        const uint32_t col0 = ((warp - 2) >> 2) * C::NC;
        uint32_t j = 0;
        for (uint32_t u = blockIdx.x; u < units; u += gridDim.x, ++j) {
            uint32_t tile, seg, m0, c_begin, n_it;
            decode(u, tile, seg, m0, c_begin, n_it);
            const uint32_t ab = j & 1, aph = (j >> 1) & 1;
            if (!__all_sync(0xffffffffu, mbar_wait(bar_tfull + 8 * ab, aph, abort_flag))) break;
            tc_fence_after();
            const uint32_t taddr = tmem_base + ((quarter * 32u) << 16) + ab * NT + col0;
            const uint32_t row = tile * 128 + quarter * 32 + lane;
#pragma unroll
            for (int c = 0; c < C::NC; c += 16) {
                const uint32_t mc = m0 + col0 + c;
                if (mc >= M) break;                                       // uniform over the warp
                int32_t v[16];
                tmem_ld<16>(taddr + c, v);
                tmem_ld_wait16(v);
                if constexpr (EPI == EPI_PARTS) {
                    if (row < N) {
                        float *dst = parts + ((size_t)seg * M + mc) * N + row;
#pragma unroll
                        for (int i = 0; i < 16; ++i) if (mc + i < M) dst[(size_t)i * N] = __int_as_float(v[i]);
                    }
                } else if constexpr (EPI == EPI_BF16) {
                    if (row < N) {
                        __nv_bfloat16 *dst = out + (size_t)mc * ldo + row;
#pragma unroll
                        for (int i = 0; i < 16; ++i) if (mc + i < M) dst[(size_t)i * ldo] = __float2bfloat16(__int_as_float(v[i]));
                    }
                } else {
                    // lanes 0-15 hold the gate sums, lanes 16-31 the up sums of the same 16 hidden indices: a pair of columns
                    // is exchanged so that the low lanes finish the even and the high lanes the odd activation row
                    const uint32_t f = tile * 64 + quarter * 16 + (lane & 15);
                    const bool hi = lane >= 16;
#pragma unroll
                    for (int i = 0; i < 16; i += 2) {
                        const float a = __int_as_float(v[i]), b = __int_as_float(v[i + 1]);
                        const float got = __shfl_xor_sync(0xffffffffu, hi ? a : b, 16);
                        const float g = hi ? got : a, up = hi ? b : got;
                        const uint32_t m = mc + i + (hi ? 1 : 0);
                        if (m < M && f < F) out[(size_t)m * ldo + f] = __float2bfloat16(qb_swiglu(g, up));
                    }
                }
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(bar_tempty + 8 * ab);
        }
    }
    tc_fence_before();
    __syncthreads();
    if (*abort_flag) {
        if (threadIdx.x == 0) atomicExch(err_flag, 4000 + (int)(blockIdx.x % 1000));
        for (int i = 0; i < 2000; ++i) __nanosleep(1000);                 // let this CTA's copies in flight land
        __syncthreads();
    }
    if (warp == 1) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(C::TMEM_COLS) : "memory");
    }
}

// Tensor maps of the activation buffers, cached per (device, buffer, shape, tile).
struct MapKey {
    int dev; const void *p; uint32_t cap, cols, ld, nt;
    bool operator<(const MapKey &o) const { return std::tie(dev, p, cap, cols, ld, nt) < std::tie(o.dev, o.p, o.cap, o.cols, o.ld, o.nt); }
};
std::map<MapKey, CUtensorMap> g_maps;
std::mutex g_map_lock;

struct GemmOut { float *parts = nullptr; __nv_bfloat16 *out = nullptr; uint32_t ldo = 0, F = 0; };

template <int NT, int EPI>
int launch_dense(qb_ctx *ctx, const QbDense &w, const QbActBuf &x, uint32_t M, const GemmOut &o, uint32_t S) {
    using C = DgCfg<NT>;
    QB_CUDA(cudaFuncSetAttribute(dense_gemm_kernel<NT, EPI>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::TOTAL));
    CUtensorMap map;
    {
        std::lock_guard<std::mutex> lock(g_map_lock);
        if (g_maps.size() > 4096) g_maps.clear();
        const MapKey key{ctx->device, x.p, x.cap, w.cols, x.ld, (uint32_t)NT};
        auto it = g_maps.find(key);
        if (it == g_maps.end()) {
            CUtensorMap m;
            QB_TRY(qb_make_tmap_2d(&m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, x.p, w.cols, x.cap, (uint64_t)x.ld * 2, 64, NT, CU_TENSOR_MAP_SWIZZLE_128B));
            it = g_maps.emplace(key, m).first;
        }
        map = it->second;
    }
    const uint32_t m_tiles = (M + NT - 1) / NT, units = (w.rows_pad / 128) * S * m_tiles;
    const uint32_t grid = std::min<uint32_t>(units, (uint32_t)ctx->sm_count * C::CTAS);
    QB_CUDA(qb_launch_pdl(ctx->stream, dense_gemm_kernel<NT, EPI>, dim3(grid), dim3(C::THREADS), (size_t)C::TOTAL, (const uint8_t *)w.rec, map, w.kc, w.rows, M,
                          o.parts, o.out, o.ldo, o.F, S, m_tiles, units, ctx->err_flag_dev));
    QB_LAUNCHED(ctx, "dense_gemm_kernel");
    return QB_OK;
}

// Activation rows per tile: the smallest that covers M up to 64 rows, else the one with the least estimated time (waves of
// units over the SMs x tile width / efficiency of the tile).
uint32_t pick_nt(const QbDense &w, uint32_t M, uint32_t sms) {
    if (M <= 16) return 16;
    if (M <= 32) return 32;
    if (M <= 64) return 64;
    uint32_t best = 64;
    double best_t = 1e300;
    const struct { uint32_t nt; double eff; } cand[] = {{64, 0.6}, {128, 0.9}, {256, 1.0}};
    for (const auto &c : cand) {
        const uint32_t units = (w.rows_pad / 128) * ((M + c.nt - 1) / c.nt);
        const double t = (double)((units + sms - 1) / sms) * c.nt / c.eff;
        if (t < best_t * 0.999) { best_t = t; best = c.nt; }
    }
    return best;
}

template <int EPI>
int launch_nt(qb_ctx *ctx, const QbDense &w, const QbActBuf &x, uint32_t M, const GemmOut &o, uint32_t S) {
    QB_REQUIRE(!x.f32 && M > 0 && M <= x.cap && S > 0 && S <= w.kc && x.ld % 8 == 0 && x.ld >= w.cols, "dense gemm: bad arguments (M %u of %u, S %u, ld %u, K %u)",
               M, x.cap, S, x.ld, w.cols);
    switch (pick_nt(w, M, (uint32_t)ctx->sm_count)) {
        case 16: return launch_dense<16, EPI>(ctx, w, x, M, o, S);
        case 32: return launch_dense<32, EPI>(ctx, w, x, M, o, S);
        case 64: return launch_dense<64, EPI>(ctx, w, x, M, o, S);
        case 128: return launch_dense<128, EPI>(ctx, w, x, M, o, S);
        default: return launch_dense<256, EPI>(ctx, w, x, M, o, S);
    }
}

// ---- fp32 activations: 64 x 64 output tile, 256 threads, 4 x 4 outputs each, K in steps of 16 --------------------------
__global__ void __launch_bounds__(256)
dense_gemm_f32_kernel(const uint8_t *__restrict__ rec, uint32_t kc, uint32_t N, uint32_t K, const float *__restrict__ x, uint32_t ldx, uint32_t M,
                      float *__restrict__ out) {
    QB_PDL_ENTER();
    __shared__ float xs[16][68], ws[16][68];
    const uint32_t tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const uint32_t n0 = blockIdx.x * 64, m0 = blockIdx.y * 64;
    float acc[4][4] = {};
    for (uint32_t k0 = 0; k0 < K; k0 += 16) {
        if (tid < 128) {                                             // 64 weight rows x two 8-column pieces
            const uint32_t r = tid >> 1, p = tid & 1;                // (row padding of the records covers r up to rows_pad)
            const uint32_t row = n0 + r, c8 = k0 / 8 + p;
            uint4 raw = make_uint4(0u, 0u, 0u, 0u);
            if (row < N && c8 < kc * 8) raw = *reinterpret_cast<const uint4 *>(rec + qb_dense_offset(kc, row, c8));
            const __nv_bfloat162 *b = reinterpret_cast<const __nv_bfloat162 *>(&raw);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float2 f = __bfloat1622float2(b[i]);
                ws[p * 8 + 2 * i][r] = f.x;
                ws[p * 8 + 2 * i + 1][r] = f.y;
            }
        }
        for (uint32_t i = tid; i < 1024; i += 256) {
            const uint32_t r = i >> 4, k = i & 15;
            xs[k][r] = (m0 + r < M && k0 + k < K) ? x[(size_t)(m0 + r) * ldx + k0 + k] : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < 16; ++k) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) { a[i] = xs[k][ty * 4 + i]; b[i] = ws[k][tx * 4 + i]; }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const uint32_t m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
            if (m < M && n < N) out[(size_t)m * N + n] = acc[i][j];
        }
}

template <typename T> __device__ __forceinline__ T act_cast(float v);
template <> __device__ __forceinline__ float act_cast<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 act_cast<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

template <typename T>
__global__ void dense_swiglu_kernel(const float *__restrict__ parts, uint32_t S, size_t pstride, uint32_t N, uint32_t M, uint32_t F, T *__restrict__ out,
                                    uint32_t ldo) {
    QB_PDL_ENTER();
    const uint32_t f = blockIdx.x * blockDim.x + threadIdx.x, m = blockIdx.y;
    if (f >= F) return;
    const size_t g = (size_t)m * N + qb_gate_col(f);
    out[(size_t)m * ldo + f] = act_cast<T>(qb_swiglu(qb_ldsum(parts, g, S, pstride), qb_ldsum(parts, g + 16, S, pstride)));
}

__global__ void dense_pack_kernel(const uint16_t *__restrict__ src, uint32_t cols, QbDenseRows rows, uint8_t *__restrict__ rec, uint32_t kc) {
    const uint64_t i = (uint64_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (uint64_t)rows.n * cols) return;
    const uint32_t r = (uint32_t)(i / cols), c = (uint32_t)(i % cols);
    *reinterpret_cast<uint16_t *>(rec + qb_dense_offset(kc, rows.dst(r), c >> 3) + (c & 7) * 2) = src[i];
}

__global__ void dense_synth_kernel(uint32_t cols, QbDenseRows rows, uint8_t *__restrict__ rec, uint32_t kc, uint64_t seed, uint32_t tensor_id, float amp) {
    const uint64_t i = (uint64_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (uint64_t)rows.n * cols) return;
    const uint32_t r = (uint32_t)(i / cols), c = (uint32_t)(i % cols);
    const float u = (float)(qs_rand_u32(seed, tensor_id, i) >> 8) * (1.0f / 8388608.0f) - 1.0f;
    *reinterpret_cast<__nv_bfloat16 *>(rec + qb_dense_offset(kc, rows.dst(r), c >> 3) + (c & 7) * 2) = __float2bfloat16(amp * u);
}

}  // namespace

int qb_dense_alloc(qb_ctx *ctx, uint32_t rows, uint32_t cols, QbDense *w) {
    QB_REQUIRE(rows > 0 && cols > 0, "dense weight: empty matrix");
    w->rows = rows; w->cols = cols;
    w->rows_pad = (rows + 127) / 128 * 128;
    w->kc = (cols + 63) / 64;
    QB_CUDA(cudaMalloc(&w->rec, w->bytes()));
    QB_CUDA(cudaMemsetAsync(w->rec, 0, w->bytes(), ctx->stream));
    return QB_OK;
}
void qb_dense_free(QbDense *w) {
    if (w->rec) cudaFree(w->rec);
    *w = QbDense();
}
int qb_dense_upload(qb_ctx *ctx, QbDense *w, const QbDenseRows &rows, const uint16_t *host) {
    QB_REQUIRE(rows.n > 0 && rows.dst(rows.n - 1) < w->rows, "dense weight: rows outside the matrix");
    const size_t n = (size_t)rows.n * w->cols;
    void *stage = nullptr;
    QB_TRY(qb_ctx_scratch(ctx, n * 2, &stage));
    QB_CUDA(cudaMemcpyAsync(stage, host, n * 2, cudaMemcpyHostToDevice, ctx->stream));
    dense_pack_kernel<<<(unsigned)((n + 255) / 256), 256, 0, ctx->stream>>>((const uint16_t *)stage, w->cols, rows, w->rec, w->kc);
    QB_LAUNCHED(ctx, "dense_pack_kernel");
    return QB_OK;
}
int qb_dense_fill_synth(qb_ctx *ctx, QbDense *w, const QbDenseRows &rows, uint64_t seed, uint32_t tensor_id, float amp) {
    QB_REQUIRE(rows.n > 0 && rows.dst(rows.n - 1) < w->rows, "dense weight: rows outside the matrix");
    const size_t n = (size_t)rows.n * w->cols;
    dense_synth_kernel<<<(unsigned)((n + 255) / 256), 256, 0, ctx->stream>>>(w->cols, rows, w->rec, w->kc, seed, tensor_id, amp);
    QB_LAUNCHED(ctx, "dense_synth_kernel");
    return QB_OK;
}

int qb_act_alloc(qb_ctx *ctx, QbActBuf *a, uint32_t rows, uint32_t cols, bool f32) {
    a->cap = rows; a->ld = (cols + 63) / 64 * 64; a->f32 = f32;
    const size_t bytes = (size_t)rows * a->ld * (f32 ? 4 : 2);
    QB_CUDA(cudaMalloc(&a->p, bytes));
    QB_CUDA(cudaMemsetAsync(a->p, 0, bytes, ctx->stream));
    return QB_OK;
}

uint32_t qb_dense_split(const QbDense &w, uint32_t M, bool f32, uint32_t sms) {
    if (f32 || M > 64) return 1;
    const uint32_t tiles = w.rows_pad / 128, slots = 2 * sms;       // not a function of M: a decode row's bits do not depend on the batch
    return std::max(1u, std::min({slots / tiles, 8u, w.kc / 4}));
}

int qb_dense_gemm(qb_ctx *ctx, const QbDense &w, const QbActBuf &x, uint32_t M, float *parts, uint32_t S) {
    if (x.f32) {
        QB_REQUIRE(S == 1 && M > 0 && M <= x.cap && x.ld >= w.cols, "dense gemm: bad arguments");
        QB_CUDA(qb_launch_pdl(ctx->stream, dense_gemm_f32_kernel, dim3((w.rows + 63) / 64, (M + 63) / 64), dim3(256), (size_t)0, (const uint8_t *)w.rec, w.kc, w.rows,
                              w.cols, (const float *)x.p, x.ld, M, parts));
        QB_LAUNCHED(ctx, "dense_gemm_f32_kernel");
        return QB_OK;
    }
    GemmOut o;
    o.parts = parts;
    return launch_nt<EPI_PARTS>(ctx, w, x, M, o, S);
}

int qb_dense_gemm_bf16(qb_ctx *ctx, const QbDense &w, const QbActBuf &x, uint32_t M, __nv_bfloat16 *out, uint32_t ld) {
    GemmOut o;
    o.out = out; o.ldo = ld;
    return launch_nt<EPI_BF16>(ctx, w, x, M, o, 1);
}

int qb_dense_gate_up(qb_ctx *ctx, const QbDense &w, const QbActBuf &x, uint32_t M, uint32_t F, float *parts, const QbActBuf &out) {
    const uint32_t S = qb_dense_split(w, M, x.f32, (uint32_t)ctx->sm_count);
    if (!x.f32 && S == 1) {
        GemmOut o;
        o.out = (__nv_bfloat16 *)out.p; o.ldo = out.ld; o.F = F;
        return launch_nt<EPI_SWIGLU>(ctx, w, x, M, o, 1);
    }
    QB_TRY(qb_dense_gemm(ctx, w, x, M, parts, S));
    const dim3 grid((F + 255) / 256, M);
    if (x.f32)
        QB_CUDA(qb_launch_pdl(ctx->stream, dense_swiglu_kernel<float>, grid, dim3(256), (size_t)0, (const float *)parts, S, (size_t)M * w.rows, w.rows, M, F,
                              (float *)out.p, out.ld));
    else
        QB_CUDA(qb_launch_pdl(ctx->stream, dense_swiglu_kernel<__nv_bfloat16>, grid, dim3(256), (size_t)0, (const float *)parts, S, (size_t)M * w.rows, w.rows, M,
                              F, (__nv_bfloat16 *)out.p, out.ld));
    QB_LAUNCHED(ctx, "dense_swiglu_kernel");
    return QB_OK;
}

// ---- op-level entry points ----------------------------------------------------------------------------------------------
namespace {
__global__ void to_bf16_kernel(const float *__restrict__ x, uint32_t stride, uint32_t K, __nv_bfloat16 *__restrict__ out, uint32_t ld) {
    const uint32_t k = blockIdx.x * blockDim.x + threadIdx.x, m = blockIdx.y;
    if (k < K) out[(size_t)m * ld + k] = __float2bfloat16(x[(size_t)m * stride + k]);
}
}  // namespace

struct qb_dense { QbDense w; };

extern "C" int qb_dense_weight(qb_ctx *ctx, const void *host_bf16, uint32_t rows, uint32_t cols, qb_dense **out) {
    QB_REQUIRE(ctx && host_bf16 && out, "qb_dense_weight: null argument");
    QB_CUDA(cudaSetDevice(ctx->device));
    auto *d = new qb_dense();
    QbDenseRows r;
    r.n = r.group = r.stride = rows;
    int st = qb_dense_alloc(ctx, rows, cols, &d->w);
    if (st == QB_OK) st = qb_dense_upload(ctx, &d->w, r, (const uint16_t *)host_bf16);
    if (st != QB_OK) { qb_dense_free(&d->w); delete d; return st; }
    *out = d;
    return QB_OK;
}
extern "C" int qb_dense_weight_synth(qb_ctx *ctx, uint64_t seed, uint32_t rows, uint32_t cols, qb_dense **out) {
    QB_REQUIRE(ctx && out, "qb_dense_weight_synth: null argument");
    QB_CUDA(cudaSetDevice(ctx->device));
    auto *d = new qb_dense();
    QbDenseRows r;
    r.n = r.group = r.stride = rows;
    int st = qb_dense_alloc(ctx, rows, cols, &d->w);
    if (st == QB_OK) st = qb_dense_fill_synth(ctx, &d->w, r, seed, 1, 0.02f);
    if (st != QB_OK) { qb_dense_free(&d->w); delete d; return st; }
    *out = d;
    return QB_OK;
}
extern "C" void qb_dense_weight_free(qb_ctx *ctx, qb_dense *d) {
    if (!d) return;
    cudaStreamSynchronize(ctx->stream);
    qb_dense_free(&d->w);
    delete d;
}
extern "C" int qb_dense_matmul(qb_ctx *ctx, const qb_dense *d, const float *x, uint32_t M, uint32_t x_stride, float *y, int f32) {
    QB_REQUIRE(ctx && d && x && y && M > 0 && x_stride >= d->w.cols, "qb_dense_matmul: bad arguments");
    QB_CUDA(cudaSetDevice(ctx->device));
    const QbDense &w = d->w;
    QbActBuf a;
    a.cap = M;
    if (f32) {
        a.p = const_cast<float *>(x); a.ld = x_stride; a.f32 = true;
        return qb_dense_gemm(ctx, w, a, M, y, 1);
    }
    const uint32_t S = qb_dense_split(w, M, false, (uint32_t)ctx->sm_count);
    a.ld = (w.cols + 63) / 64 * 64;
    QB_TRY(qb_ctx_scratch2(ctx, (size_t)M * a.ld * 2, &a.p));
    to_bf16_kernel<<<dim3((w.cols + 255) / 256, M), 256, 0, ctx->stream>>>(x, x_stride, w.cols, (__nv_bfloat16 *)a.p, a.ld);
    QB_LAUNCHED(ctx, "to_bf16_kernel");
    if (S == 1) return qb_dense_gemm(ctx, w, a, M, y, 1);
    void *parts = nullptr;
    QB_TRY(qb_ctx_scratch(ctx, (size_t)S * M * w.rows * sizeof(float), &parts));
    QB_TRY(qb_dense_gemm(ctx, w, a, M, (float *)parts, S));
    return qb_launch_reduce_parts(ctx, (const float *)parts, S, M, w.rows, y, w.rows);
}
