// Absorbed latent attention on the 5th-generation tensor cores: the spans of latent_split_kernel (latent_attention.cu) with
// tcgen05.mma, accumulators in tensor memory and the cached latents by TMA.
//
// All heads of a sequence's rows attend the same vectors, so the keys are the MMA's M dimension and the (row, head) queries
// its N dimension, and one shared-memory tile of 128 cached vectors is both operands:
//     S^T [128 keys x NQ]   = tile [128 x pitch] . Qa^T       (A K-major, as the cache lies; pitch = latent + shared key part)
//     O^T [rank x NQ]      += tile^T [rank x 128] . P^T       (A MN-major, the latent columns of the same tile, 128 at a time)
// A tile is NU units of 64 columns (16 KB each) at fixed places; the columns of the shared key part are free again after the
// scores, the latent columns pair by pair as the value products pass over them, and the next tile is loaded behind them.
// A key is a TMEM lane and a thread (times NQ / 16 threads of 16 query columns each).  The running maximum of a column is
// exact; when it grows, the threads of that column group rescale their part of O in tensor memory (tcgen05.ld, multiply,
// tcgen05.st) before they release the tile's weights.  Row sums stay per key lane until the end of the span.
//
// Warp 0 loads, warp 1 issues the MMAs and owns the tensor memory, the others are softmax threads and write the span out.
// Every wait is bounded (error flag).  No multicast.
#include "layered.h"
#include "tc_common.cuh"

#include <mutex>

namespace {
using namespace qbtc;

constexpr uint32_t KT = 128, UNIT = KT * 128;       // keys of a tile; bytes of a 64-column unit
constexpr float LOG2E = 1.4426950408889634f;

template <int NQ>
struct LtcCfg {
    static constexpr int SM_THREADS = NQ * 8;       // softmax threads: 128 lanes x NQ / 16 column groups
    static constexpr int THREADS = 64 + SM_THREADS;
    static constexpr int CTAS = NQ <= 16 ? 3 : NQ <= 32 ? 2 : 1;      // resident CTAs per SM that the registers allow (small tiles)
    static constexpr uint32_t OST = NQ <= 32 ? 32 : 64;      // column stride of S and of the blocks of O in tensor memory
};
struct LtcSmem { uint32_t q, p, misc, total; };
__host__ __device__ inline LtcSmem ltc_smem(uint32_t NU, uint32_t NQ) {
    LtcSmem m;
    m.q = NU * UNIT;
    m.p = m.q + NU * NQ * 128;
    m.misc = m.p + 2 * NQ * 128;
    m.total = m.misc + 512 + NQ * 4 + 2 * NQ * 16 + 1024;      // + slack to align the base to 1024
    return m;
}
__host__ __device__ inline uint32_t ltc_tmem_cols(uint32_t NB, uint32_t ost) {
    const uint32_t need = (1 + NB) * ost;
    return need <= 64 ? 64 : need <= 128 ? 128 : need <= 256 ? 256 : 512;
}

// grid (spans, query groups, sequences)
template <int NQ>
__global__ void __launch_bounds__(LtcCfg<NQ>::THREADS, LtcCfg<NQ>::CTAS)
latent_split_tc_kernel(QbLatent a, const __grid_constant__ CUtensorMap map, uint32_t n_splits, uint32_t NU, uint32_t NB) {
    using C = LtcCfg<NQ>;
    extern __shared__ uint8_t smem_raw[];
    uint8_t *smem = reinterpret_cast<uint8_t *>(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    const LtcSmem L = ltc_smem(NU, NQ);
    uint8_t *misc = smem + L.misc;
    const uint32_t NG = NB + (NU > 2 * NB ? 1 : 0);                     // groups of units: NB pairs of latent columns, the rest
    // barriers: full[9], empty[9], scores, weights, output
    const uint32_t bar_full = smem_u32(misc), bar_empty = bar_full + 72, bar_s = bar_empty + 72, bar_p = bar_s + 8, bar_o = bar_p + 8;
    uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(misc + 192);
    volatile int *abort_flag = reinterpret_cast<volatile int *>(misc + 196);
    int *qpos = reinterpret_cast<int *>(misc + 512);                    // [NQ]
    float *red = reinterpret_cast<float *>(misc + 512 + NQ * 4);        // [2][NQ][4 lane quarters]
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const uint32_t cols = ltc_tmem_cols(NB, C::OST);
    if (tid == 0) {
        for (uint32_t i = 0; i < 9; ++i) { mbar_init(bar_full + 8 * i, 1); mbar_init(bar_empty + 8 * i, 1); }
        mbar_init(bar_s, 1);
        mbar_init(bar_p, C::SM_THREADS);
        mbar_init(bar_o, 1);
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        asm volatile("prefetch.tensormap [%0];" ::"l"(reinterpret_cast<uint64_t>(&map)) : "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(cols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_s = *tmem_slot, tmem_o = tmem_s + C::OST;
    // only now, with this CTA's tensor memory in hand: a dependent kernel that allocates some cannot get in its way
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    asm volatile("griddepcontrol.wait;" ::: "memory");

    const uint32_t split = blockIdx.x, sg = blockIdx.z, s = sg / a.groups, grp = sg % a.groups, hg = a.heads_per_group(), nq = a.R * hg, qg = blockIdx.y * NQ;
    const int base = a.seq_pos[s];
    const uint32_t span = qb_latent_span((uint32_t)base + a.R, a.max_splits);
    const uint32_t q_last = min(qg + NQ, nq) - 1;
    const int k_begin = (int)(split * span), k_end = min(k_begin + (int)span, base + (int)(q_last / hg) + 1);
    const uint32_t n_tiles = k_begin < k_end ? (uint32_t)(k_end - k_begin + KT - 1) / KT : 0;      // 0: nothing visible (uniform)
    // Loads of tile t: lane & 7 names a page of the tile, `slot` its first slot.
    auto load_tile = [&](uint32_t t) -> bool {
        const int32_t *pt = a.page_table + (size_t)s * a.pt_stride;
        const int pg0 = (k_begin + (int)(t * KT)) >> 4, pg_last = (k_end - 1) >> 4;      // 16-key pages (checked by the launcher)
        // pages past the last key are not looked up: the last valid one is loaded again (finite values, masked)
        const int slot = max(0, pt[min(min(pg0 + (int)(lane & 7), pg_last), (int)a.pt_stride - 1)]) * 16;
        for (uint32_t gi = 0; gi < NG; ++gi) {
            const uint32_t g = NG > NB ? (gi == 0 ? NB : gi - 1) : gi, u0 = 2 * g, un = g < NB ? 2 : NU - 2 * NB;
            if (!__all_sync(0xffffffffu, mbar_wait_idle(bar_empty + 8 * g, (t & 1) ^ 1, abort_flag, 50))) return false;
            const uint32_t full = bar_full + 8 * g;
            if (lane == 0) mbar_expect_tx(full, un * UNIT);
            __syncwarp();
            for (uint32_t i = lane; i < un * 8; i += 32) {               // (i & 7 == lane & 7)
                const uint32_t u = u0 + (i >> 3);
                tma_load_2d(smem_u32(smem + u * UNIT) + (i & 7) * 2048, &map, (int)(grp * a.pitch() + u * 64), slot, full);
            }
        }
        return true;
    };
    if (n_tiles && warp == 0) load_tile(0);                              // under way while the queries are staged
    if (n_tiles) {
        // queries in the swizzled K-major operand layout: [unit][NQ rows][128 B]; columns past the pitch and rows past the last query zero
        const uint32_t D = a.pitch();
        const __nv_bfloat16 *qa = (const __nv_bfloat16 *)a.qa + ((size_t)sg * nq + qg) * D;
        for (uint32_t i = tid; i < NQ * NU * 8; i += C::THREADS) {
            const uint32_t q = i / (NU * 8), c8 = i % (NU * 8);
            uint4 v = make_uint4(0u, 0u, 0u, 0u);
            if (qg + q < nq && c8 * 8 < D) v = *reinterpret_cast<const uint4 *>(qa + (size_t)q * D + c8 * 8);
            *reinterpret_cast<uint4 *>(smem + L.q + (c8 >> 3) * (NQ * 128) + q * 128 + (((c8 & 7) ^ (q & 7)) << 4)) = v;
        }
        if (tid < NQ) qpos[tid] = qg + tid < nq ? base + (int)((qg + tid) / hg) : -1;
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();

    if (n_tiles == 0) {
        // nothing to do
    } else if (warp == 0) {
        for (uint32_t t = 1; t < n_tiles; ++t)
            if (!load_tile(t)) break;
    } else if (warp == 1) {
        if (lane == 0) {
            // D fp32, A = B = bf16, N = NQ, M = 128; the value products read A MN-major
            constexpr uint32_t idesc_s = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(NQ >> 3) << 17) | ((128u >> 4) << 24);
            constexpr uint32_t idesc_o = idesc_s | (1u << 15);
            const uint32_t tile = smem_u32(smem), q_addr = tile + L.q, p_addr = tile + L.p;
            bool ok = true;
            for (uint32_t t = 0; t < n_tiles && ok; ++t) {
                uint32_t acc = 0;
                for (uint32_t gi = 0; gi < NG; ++gi) {
                    const uint32_t g = NG > NB ? (gi == 0 ? NB : gi - 1) : gi, un = g < NB ? 2 : NU - 2 * NB;
                    if (!mbar_wait(bar_full + 8 * g, t & 1, abort_flag)) { ok = false; break; }
                    tc_fence_after();
                    for (uint32_t u = 2 * g; u < 2 * g + un; ++u)
#pragma unroll
                        for (int ks = 0; ks < 4; ++ks, acc = 1)
                            tc_mma_f16(tmem_s, smem_desc_sw128(tile + u * UNIT + ks * 32), smem_desc_sw128(q_addr + u * (NQ * 128) + ks * 32), idesc_s, acc);
                    if (g == NB) tc_commit(bar_empty + 8 * g);
                }
                if (!ok) break;
                tc_commit(bar_s);
                if (!mbar_wait(bar_p, t & 1, abort_flag)) break;
                tc_fence_after();
                for (uint32_t b = 0; b < NB; ++b) {
#pragma unroll
                    for (int ks = 0; ks < 8; ++ks)
                        tc_mma_f16(tmem_o + b * C::OST, smem_desc_mn_sw128(tile + 2 * b * UNIT + ks * 2048, UNIT),
                                   smem_desc_sw128(p_addr + (ks / 4) * (NQ * 128) + (ks % 4) * 32), idesc_o, (t > 0 || ks > 0) ? 1u : 0u);
                    tc_commit(bar_empty + 8 * b);
                }
                if (t + 1 == n_tiles) tc_commit(bar_o);
            }
        }
    } else {
        const uint32_t quarter = warp & 3, q0 = ((warp - 2) >> 2) * 16, r = quarter * 32 + lane;      // key lane, first query column
        const uint32_t lane_addr = (quarter * 32u) << 16;
        // factor of a key's scores, looked up a tile ahead
        const float sl0 = a.scale * LOG2E;
        auto key_factor = [&](uint32_t t) -> float {
            const int key = k_begin + (int)(t * KT + r);
            if (!a.key_scale || key >= k_end) return sl0;
            const int64_t at = qb_latent_slot(a, a.page_table + (size_t)s * a.pt_stride, (uint32_t)key);
            return at < 0 ? 0.0f : sl0 * a.key_scale[(size_t)at * a.groups + grp];
        };
        float sl_next = key_factor(0);
        const float4 *red4 = reinterpret_cast<const float4 *>(red);
        uint8_t *prow = smem + L.p + (r >> 6) * (NQ * 128) + (r & 7) * 2;
        const uint32_t ch = (r & 63) >> 3;
        float mx[16], sum[16];
#pragma unroll
        for (int j = 0; j < 16; ++j) { mx[j] = -INFINITY; sum[j] = 0.0f; }
        bool ok = true;
        for (uint32_t t = 0; t < n_tiles; ++t) {
            // a wait that ran out does not leave the loop: the warps of a column group meet at its named barrier either way, and
            // the waits that follow return at once
            ok = __all_sync(0xffffffffu, mbar_wait_idle(bar_s, t & 1, abort_flag, 20)) && ok;
            tc_fence_after();
            uint32_t raw[16];
            tmem_ld16(tmem_s + lane_addr + q0, raw);
            tmem_wait_dep(raw);
            const int key = k_begin + (int)(t * KT + r);
            const float sl = sl_next;
            if (t + 1 < n_tiles) sl_next = key_factor(t + 1);
            float sc[16], cm[16];
#pragma unroll
            for (int j = 0; j < 16; ++j) {
                sc[j] = key <= qpos[q0 + j] && key < k_end ? __uint_as_float(raw[j]) * sl : -INFINITY;
                cm[j] = sc[j];
            }
            const float wmax = lane_transpose_reduce16<true>(cm, lane);       // lanes j, j + 16: column q0 + j over this warp's keys
            const uint32_t rb = (t & 1) * NQ;
            if (lane < 16) red[(rb + q0 + lane) * 4 + quarter] = wmax;
            asm volatile("bar.sync %0, 128;" ::"r"(1 + q0 / 16) : "memory");   // the four warps of a column group
            bool grew = false;
            float alpha[16];
#pragma unroll
            for (int j = 0; j < 16; ++j) {
                const float4 m4 = red4[rb + q0 + j];
                const float nm = fmaxf(mx[j], fmaxf(fmaxf(m4.x, m4.y), fmaxf(m4.z, m4.w)));
                grew |= nm > mx[j];
                const float ref = nm == -INFINITY ? 0.0f : nm;
                alpha[j] = exp2f(mx[j] - ref);
                mx[j] = nm;
                const __nv_bfloat16 p = __float2bfloat16(exp2f(sc[j] - ref));
                sum[j] = fmaf(sum[j], alpha[j], __bfloat162float(p));         // the rounded weights, as the tensor cores see them
                const uint32_t q = q0 + j;
                *reinterpret_cast<__nv_bfloat16 *>(prow + q * 128 + ((ch ^ (q & 7)) << 4)) = p;
            }
            // (bar_s says that the previous tile's value products are done: O may be rescaled, and P was free)
            if (t > 0 && grew)                                                   // uniform over the column group
                for (uint32_t b = 0; b < NB; ++b) {
                    uint32_t o[16];
                    const uint32_t at = tmem_o + b * C::OST + lane_addr + q0;
                    tmem_ld16(at, o);
                    tmem_wait_dep(o);
#pragma unroll
                    for (int j = 0; j < 16; ++j) o[j] = __float_as_uint(__uint_as_float(o[j]) * alpha[j]);
                    tmem_st16(at, o);
                }
            tmem_st_wait();
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            tc_fence_before();
            mbar_arrive(bar_p);
        }
        ok = __all_sync(0xffffffffu, mbar_wait_idle(bar_o, 0, abort_flag, 20)) && ok;
        tc_fence_after();
        const float wsum = lane_transpose_reduce16<false>(sum, lane);
        const uint32_t rb = (n_tiles & 1) * NQ;
        if (lane < 16) red[(rb + q0 + lane) * 4 + quarter] = wsum;
        asm volatile("bar.sync %0, 128;" ::"r"(1 + q0 / 16) : "memory");
        if (ok) {
            const size_t row0 = (size_t)sg * nq + qg + q0;
            if (quarter == 0 && lane < 16 && qg + q0 + lane < nq) {
                const float4 l4 = red4[rb + q0 + lane];
                float m = mx[0];
#pragma unroll
                for (int j = 1; j < 16; ++j) m = lane == (uint32_t)j ? mx[j] : m;
                float *ml = a.part_ml + ((row0 + lane) * n_splits + split) * 2;
                ml[0] = m / LOG2E;                                              // natural units, as the merge takes them
                ml[1] = ((l4.x + l4.y) + l4.z) + l4.w;
            }
            for (uint32_t b = 0; b < NB; ++b) {
                uint32_t o[16];
                tmem_ld16(tmem_o + b * C::OST + lane_addr + q0, o);
                tmem_wait_dep(o);
                const uint32_t c = b * 128 + r;
#pragma unroll
                for (int j = 0; j < 16; ++j)
                    if (c < a.rank && qg + q0 + j < nq) a.part_acc[((row0 + j) * n_splits + split) * a.rank + c] = __uint_as_float(o[j]);
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (*abort_flag) {
        if (tid == 0) atomicExch(a.err_flag, 5000 + (int)(blockIdx.x % 1000));
        for (int i = 0; i < 2000; ++i) __nanosleep(1000);                       // let this CTA's copies in flight land
        __syncthreads();
    }
    if (warp == 1) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_s), "r"(cols) : "memory");
    }
}

struct MapKey {
    int dev; const void *p; uint64_t slots; uint32_t cols;
    bool operator<(const MapKey &o) const { return std::tie(dev, p, slots, cols) < std::tie(o.dev, o.p, o.slots, o.cols); }
};
std::map<MapKey, CUtensorMap> g_maps;
std::mutex g_lock;

template <int NQ>
int launch(qb_ctx *ctx, const QbLatent &a, uint32_t n_splits, uint32_t NU, uint32_t NB) {
    const uint32_t smem = ltc_smem(NU, NQ).total;
    QB_CUDA(cudaFuncSetAttribute(latent_split_tc_kernel<NQ>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    CUtensorMap map;
    {
        std::lock_guard<std::mutex> lock(g_lock);
        if (g_maps.size() > 4096) g_maps.clear();
        const uint32_t cols = a.groups * a.pitch();
        const MapKey key{ctx->device, a.cache, a.slots, cols};
        auto it = g_maps.find(key);
        if (it == g_maps.end()) {
            CUtensorMap m;
            // a box: one 128-byte column of a 16-key page; columns past a vector read as the next group's (their queries are zero),
            // past the last as zero
            QB_TRY(qb_make_tmap_2d(&m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, a.cache, cols, a.slots, (uint64_t)cols * 2, 64, 16, CU_TENSOR_MAP_SWIZZLE_128B));
            it = g_maps.emplace(key, m).first;
        }
        map = it->second;
    }
    QB_CUDA(qb_launch_pdl(ctx->stream, latent_split_tc_kernel<NQ>, dim3(n_splits, (a.group_queries() + NQ - 1) / NQ, a.ns * a.groups), dim3(LtcCfg<NQ>::THREADS), (size_t)smem, a, map,
                          n_splits, NU, NB));
    QB_LAUNCHED(ctx, "latent_split_tc_kernel");
    return QB_OK;
}

// 64-column units of a tile (the latent columns go in pairs; a unit past the vector holds columns nobody uses).
uint32_t units_of(const QbLatent &a) { return std::max((a.pitch() + 63) / 64, (a.rankp() + 127) / 128 * 2); }

// Queries per CTA: the fewest groups, then the smallest tile; 0 when the shape does not fit.
uint32_t pick_nq(const QbLatent &a) {
    const uint32_t NU = units_of(a), NB = (a.rankp() + 127) / 128, nq = a.group_queries();
    if (a.f32 || a.page_size != 16 || NB > 4) return 0;
    uint32_t best = 0;
    for (uint32_t n : {16u, 32u, 48u}) {
        if (ltc_smem(NU, n).total > 232448) continue;
        if (!best || (nq + n - 1) / n < (nq + best - 1) / best) best = n;
    }
    return best;
}

}  // namespace

bool qb_latent_tc_supports(const QbLatent &a) { return pick_nq(a) != 0; }

int qb_launch_latent_split_tc(qb_ctx *ctx, const QbLatent &a, uint32_t n_splits) {
    const uint32_t NU = units_of(a), NB = (a.rankp() + 127) / 128;
    switch (pick_nq(a)) {
        case 16: return launch<16>(ctx, a, n_splits, NU, NB);
        case 32: return launch<32>(ctx, a, n_splits, NU, NB);
        default: return launch<48>(ctx, a, n_splits, NU, NB);
    }
}
