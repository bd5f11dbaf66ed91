// Prompt rows of attention whose values are its keys, on the 5th-generation tensor cores: one pass over the keys, no spans.
//
// A CTA takes 128 (row, head) queries of one key/value head and walks the keys in tiles of 128 cached vectors:
//     S [128 queries x 128 keys]  = Q . tile^T       (both K-major; two buffers in tensor memory)
//     O [128 queries x dim]      += P . tile          (P K-major from shared memory, the value columns of the same tile MN-major)
// While the softmax threads work on one tile's scores, the tensor cores compute the next tile's; the tiles come by TMA page by
// page into two buffers where they fit.  256 softmax threads, two per query row (64 keys each).  The running maximum starts at 0,
// the score of the sink, whose share opens the sum at 1; it moves only when it is outgrown by 2^8, so O is rescaled (in
// tensor memory) a few times at most.  The epilogue divides, gates and writes the rows.
//
// Warp 0 loads, warp 1 issues the MMAs and owns the tensor memory.  Every wait is bounded (error flag).  No multicast.
#include "layered.h"
#include "tc_common.cuh"

#include <mutex>

namespace {
using namespace qbtc;

constexpr uint32_t KT = 128, UNIT = KT * 128;       // keys of a tile and queries of a CTA; bytes of a 64-column unit
constexpr uint32_t SM_THREADS = 256, THREADS = 64 + SM_THREADS, TMEM_COLS = 512, O_COL = 256;
constexpr float LOG2E = 1.4426950408889634f, SLACK = 8.0f;

struct PfSmem { uint32_t k, p, misc, total; };
__host__ __device__ inline PfSmem pf_smem(uint32_t NU, uint32_t stages) {
    PfSmem m;
    m.k = NU * UNIT;
    m.p = m.k + stages * NU * UNIT;
    m.misc = m.p + 2 * UNIT;
    m.total = m.misc + 256 + 2 * KT * 4 + 2 * 2 * KT * 4 + 1024;       // barriers, key factors, row exchange, slack to align the base
    return m;
}

// grid (sequences x key/value heads, query tiles)
__global__ void __launch_bounds__(THREADS, 1)
shared_kv_prefill_kernel(QbSharedKv a, const __grid_constant__ CUtensorMap map, uint32_t NU, uint32_t stages) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t *smem = reinterpret_cast<uint8_t *>(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    const QbLatent &L = a.at;
    const PfSmem M = pf_smem(NU, stages);
    uint8_t *misc = smem + M.misc;
    // barriers: tile full[2], tile empty[2], scores[2], weights, output
    const uint32_t bar_kf = smem_u32(misc), bar_ke = bar_kf + 16, bar_s = bar_ke + 16, bar_p = bar_s + 16, bar_o = bar_p + 8;
    uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(misc + 128);
    volatile int *abort_flag = reinterpret_cast<volatile int *>(misc + 132);
    float *kf = reinterpret_cast<float *>(misc + 256);                     // [2][KT] factor of a key's scores
    float *xch = kf + 2 * KT;                                              // [2][2][KT] row maxima (then sums) of the two halves
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    if (tid == 0) {
        for (uint32_t i = 0; i < 2; ++i) { mbar_init(bar_kf + 8 * i, 1); mbar_init(bar_ke + 8 * i, 1); mbar_init(bar_s + 8 * i, 1); }
        mbar_init(bar_p, SM_THREADS);
        mbar_init(bar_o, 1);
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        asm volatile("prefetch.tensormap [%0];" ::"l"(reinterpret_cast<uint64_t>(&map)) : "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(TMEM_COLS) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    // only now, with this CTA's tensor memory in hand: a dependent kernel that allocates some cannot get in its way
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    asm volatile("griddepcontrol.wait;" ::: "memory");

    const uint32_t sg = blockIdx.x, s = sg / L.groups, grp = sg % L.groups, hg = L.heads_per_group(), nq = L.R * hg;
    const uint32_t qg = (gridDim.y - 1 - blockIdx.y) * KT;                 // the tiles with the most keys start first
    const int base = L.seq_pos[s];
    const int k_end = base + (int)((min(qg + KT, nq) - 1) / hg) + 1;       // keys that the last query sees
    const int full_end = base + (int)(qg / hg) + 1;                        // ... that every query sees
    const uint32_t n_tiles = (uint32_t)(k_end + (int)KT - 1) / KT;
    const int32_t *pt = L.page_table + (size_t)s * L.pt_stride;
    auto key_factor = [&](uint32_t t, uint32_t r) -> float {
        const int key = (int)(t * KT + r);
        if (key >= k_end) return 0.0f;
        const int64_t at = qb_latent_slot(L, pt, (uint32_t)key);
        return at < 0 ? 0.0f : L.scale * LOG2E * L.key_scale[(size_t)at * L.groups + grp];
    };
    // Loads of tile t: lane & 7 names a page of the tile (16-key pages, checked by the launcher), `slot` its first slot.
    auto load_tile = [&](uint32_t t) -> bool {
        const uint32_t st = t % stages;
        const int pg_last = (k_end - 1) >> 4;
        // pages past the last key are not looked up: the last valid one is loaded again (finite values, masked)
        const int slot = max(0, pt[min(min((int)(t * 8 + (lane & 7)), pg_last), (int)L.pt_stride - 1)]) * 16;
        if (!__all_sync(0xffffffffu, mbar_wait_idle(bar_ke + 8 * st, ((t / stages) & 1) ^ 1, abort_flag, 20))) return false;
        const uint32_t full = bar_kf + 8 * st;
        if (lane == 0) mbar_expect_tx(full, NU * UNIT);
        __syncwarp();
        for (uint32_t i = lane; i < NU * 8; i += 32)                        // (i & 7 == lane & 7)
            tma_load_2d(smem_u32(smem + M.k + (st * NU + (i >> 3)) * UNIT) + (i & 7) * 2048, &map, (int)(grp * L.pitch() + (i >> 3) * 64), slot, full);
        return true;
    };
    if (warp == 0) load_tile(0);                                            // under way while the queries are staged
    {
        // queries in the swizzled K-major operand layout; columns past the vector and rows past the last query zero
        const uint32_t D = L.pitch(), U8 = NU * 8;
        const __nv_bfloat16 *qa = (const __nv_bfloat16 *)L.qa + ((size_t)sg * nq + qg) * D;
        for (uint32_t i = tid; i < KT * U8; i += THREADS) {
            const uint32_t q = i / U8, c8 = i % U8;
            uint4 v = make_uint4(0u, 0u, 0u, 0u);
            if (qg + q < nq && c8 * 8 < D) v = *reinterpret_cast<const uint4 *>(qa + (size_t)q * D + c8 * 8);
            *reinterpret_cast<uint4 *>(smem + (c8 >> 3) * UNIT + q * 128 + (((c8 & 7) ^ (q & 7)) << 4)) = v;
        }
        if (tid >= 64 && tid < 64 + KT) kf[tid - 64] = key_factor(0, tid - 64);
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();

    if (warp == 0) {
        for (uint32_t t = 1; t < n_tiles; ++t)
            if (!load_tile(t)) break;
    } else if (warp == 1) {
        if (lane == 0) {
            // D fp32, A = B = bf16, M = 128; scores: N = 128, both K-major; values: N = padded head size, B MN-major
            constexpr uint32_t idesc_b = (1u << 4) | (1u << 7) | (1u << 10) | ((128u >> 4) << 24), idesc_s = idesc_b | ((KT >> 3) << 17);
            const uint32_t idesc_o = idesc_b | ((L.rankp() >> 3) << 17) | (1u << 16);
            const uint32_t q_addr = smem_u32(smem), k_addr = q_addr + M.k, p_addr = q_addr + M.p;
            bool ok = true;
            auto scores = [&](uint32_t t) {
                const uint32_t st = t % stages;
                if (!(ok = mbar_wait(bar_kf + 8 * st, (t / stages) & 1, abort_flag))) return;
                tc_fence_after();
                for (uint32_t u = 0; u < NU; ++u)
#pragma unroll
                    for (int ks = 0; ks < 4; ++ks)
                        tc_mma_f16(tmem + (t & 1) * KT, smem_desc_sw128(q_addr + u * UNIT + ks * 32), smem_desc_sw128(k_addr + (st * NU + u) * UNIT + ks * 32),
                                   idesc_s, (u > 0 || ks > 0) ? 1u : 0u);
                tc_commit(bar_s + 8 * (t & 1));
            };
            scores(0);
            for (uint32_t t = 0; t < n_tiles && ok; ++t) {
                // the buffer of tile t + 1's scores was read before the weights of tile t - 1 were released
                if (stages == 2 && t + 1 < n_tiles) { scores(t + 1); if (!ok) break; }
                if (!mbar_wait(bar_p, t & 1, abort_flag)) break;
                tc_fence_after();
                const uint32_t v_addr = k_addr + (t % stages) * NU * UNIT;
#pragma unroll
                for (int ks = 0; ks < 8; ++ks)
                    tc_mma_f16(tmem + O_COL, smem_desc_sw128(p_addr + (ks / 4) * UNIT + (ks % 4) * 32), smem_desc_mn_sw128(v_addr + ks * 2048, UNIT), idesc_o,
                               (t > 0 || ks > 0) ? 1u : 0u);
                tc_commit(bar_ke + 8 * (t % stages));
                tc_commit(bar_o);
                if (stages == 1 && t + 1 < n_tiles) scores(t + 1);
            }
        }
    } else {
        const uint32_t quarter = warp & 3, half = (warp - 2) >> 2, r = quarter * 32 + lane;      // query row; which 64 keys of a tile
        const uint32_t lane_addr = (quarter * 32u) << 16, rp = L.rankp();
        const int qpos = qg + r < nq ? base + (int)((qg + r) / hg) : -1;
        uint8_t *prow = smem + M.p + half * UNIT + r * 128;
        float m = 0.0f, sum = half == 0 ? 1.0f : 0.0f;                      // the sink
        bool ok = true;
        for (uint32_t t = 0; t < n_tiles; ++t) {
            const float kf_next = half == 0 && t + 1 < n_tiles ? key_factor(t + 1, r) : 0.0f;
            // a wait that ran out does not leave the loop: the softmax warps meet at their named barrier either way
            ok = __all_sync(0xffffffffu, mbar_wait(bar_s + 8 * (t & 1), (t >> 1) & 1, abort_flag)) && ok;
            tc_fence_after();
            uint32_t v[4][16];
#pragma unroll
            for (int c = 0; c < 4; ++c) tmem_ld16(tmem + lane_addr + (t & 1) * KT + half * 64 + c * 16, v[c]);
#pragma unroll
            for (int c = 0; c < 4; ++c) tmem_wait_dep(v[c]);
            const float4 *f4 = reinterpret_cast<const float4 *>(kf + (t & 1) * KT + half * 64);
            const int key0 = (int)(t * KT + half * 64);
            const bool whole = (int)((t + 1) * KT) <= full_end;
            float mx = -INFINITY;
#pragma unroll
            for (int c = 0; c < 4; ++c)
#pragma unroll
                for (int j = 0; j < 16; j += 4) {
                    const float4 f = f4[c * 4 + j / 4];
                    const float ff[4] = {f.x, f.y, f.z, f.w};
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        float x = __uint_as_float(v[c][j + i]) * ff[i];
                        if (!whole && key0 + c * 16 + j + i > qpos) x = -INFINITY;
                        v[c][j + i] = __float_as_uint(x);
                        mx = fmaxf(mx, x);
                    }
                }
            float *x2 = xch + (t & 1) * 2 * KT;
            x2[half * KT + r] = mx;
            if (half == 0 && t + 1 < n_tiles) kf[((t + 1) & 1) * KT + r] = kf_next;      // (the last reader of that buffer was tile t - 1)
            asm volatile("bar.sync 1, 256;" ::: "memory");
            mx = fmaxf(mx, x2[(half ^ 1) * KT + r]);
            const bool grew = mx > m + SLACK;
            const float alpha = grew ? exp2f(m - mx) : 1.0f;
            if (grew) m = mx;
            sum *= alpha;
            uint32_t p[32];
#pragma unroll
            for (int c = 0; c < 4; ++c)
#pragma unroll
                for (int j = 0; j < 16; j += 2) {
                    const __nv_bfloat162 b = __floats2bfloat162_rn(exp2f(__uint_as_float(v[c][j]) - m), exp2f(__uint_as_float(v[c][j + 1]) - m));
                    const float2 f = __bfloat1622float2(b);                  // the rounded weights, as the tensor cores see them
                    sum += f.x + f.y;
                    p[c * 8 + j / 2] = *reinterpret_cast<const uint32_t *>(&b);
                }
            if (t > 0) ok = __all_sync(0xffffffffu, mbar_wait(bar_o, (t - 1) & 1, abort_flag)) && ok;      // P is free, O at rest
            tc_fence_after();
#pragma unroll
            for (int c = 0; c < 8; ++c)
                *reinterpret_cast<uint4 *>(prow + ((c ^ (r & 7)) << 4)) = make_uint4(p[4 * c], p[4 * c + 1], p[4 * c + 2], p[4 * c + 3]);
            if (t > 0 && __any_sync(0xffffffffu, grew))
                for (uint32_t c = half * 16; c < rp; c += 32) {
                    uint32_t o[16];
                    tmem_ld16(tmem + O_COL + lane_addr + c, o);
                    tmem_wait_dep(o);
#pragma unroll
                    for (int j = 0; j < 16; ++j) o[j] = __float_as_uint(__uint_as_float(o[j]) * alpha);
                    tmem_st16(tmem + O_COL + lane_addr + c, o);
                }
            tmem_st_wait();
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            tc_fence_before();
            mbar_arrive(bar_p);
        }
        ok = __all_sync(0xffffffffu, mbar_wait(bar_o, (n_tiles - 1) & 1, abort_flag)) && ok;
        tc_fence_after();
        float *x2 = xch + (n_tiles & 1) * 2 * KT;
        x2[half * KT + r] = sum;
        asm volatile("bar.sync 1, 256;" ::: "memory");
        sum += x2[(half ^ 1) * KT + r];
        const uint32_t q = qg + r, mrow = s * L.R + q / hg, h = grp * hg + q % hg;
        const bool in = ok && q < nq;
        float gate = 0.0f;
        if (in) gate = qb_sigmoid(qb_sum8(a.proj, (size_t)mrow * a.stride + (size_t)(L.H + L.groups) * L.rank + h, a.S, (size_t)L.ns * L.R * a.stride)) / sum;
        __nv_bfloat16 *out = (__nv_bfloat16 *)L.out.p + (size_t)mrow * L.out.ld + (size_t)h * L.rank;
        const bool vec = L.rank % 8 == 0;                                    // (rows of the output buffer are 16-byte aligned)
        for (uint32_t c = half * 16; c < rp; c += 32) {
            uint32_t o[16];
            tmem_ld16(tmem + O_COL + lane_addr + c, o);
            tmem_wait_dep(o);
#pragma unroll
            for (int j = 0; j < 16; j += 8) {
                if (in && vec && c + j < L.rank) {
                    uint32_t w[4];
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const __nv_bfloat162 b = __floats2bfloat162_rn(__uint_as_float(o[j + 2 * i]) * gate, __uint_as_float(o[j + 2 * i + 1]) * gate);
                        w[i] = *reinterpret_cast<const uint32_t *>(&b);
                    }
                    *reinterpret_cast<uint4 *>(out + c + j) = make_uint4(w[0], w[1], w[2], w[3]);
                } else if (in && !vec) {
#pragma unroll
                    for (int i = 0; i < 8; ++i)
                        if (c + j + i < L.rank) out[c + j + i] = __float2bfloat16(__uint_as_float(o[j + i]) * gate);
                }
            }
            __syncwarp();
        }
    }
    tc_fence_before();
    __syncthreads();
    if (*abort_flag) {
        if (tid == 0) atomicExch(L.err_flag, 7000 + (int)(blockIdx.y % 1000));
        for (int i = 0; i < 2000; ++i) __nanosleep(1000);                    // let this CTA's copies in flight land
        __syncthreads();
    }
    if (warp == 1) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(TMEM_COLS) : "memory");
    }
}

constexpr uint32_t SMEM_LIMIT = 232448;
uint32_t units_of(const QbLatent &a) { return std::max((a.pitch() + 63) / 64, (a.rankp() + 63) / 64); }

struct MapKey {
    int dev; const void *p; uint64_t slots; uint32_t cols;
    bool operator<(const MapKey &o) const { return std::tie(dev, p, slots, cols) < std::tie(o.dev, o.p, o.slots, o.cols); }
};
std::map<MapKey, CUtensorMap> g_maps;
std::mutex g_lock;

}  // namespace

bool qb_shared_kv_prefill_supports(const QbLatent &a, uint32_t sms) {
    if (a.f32 || a.page_size != 16 || a.rankp() > 256 || pf_smem(units_of(a), 1).total > SMEM_LIMIT) return false;
    // enough queries to fill a tile, and enough CTAs unless the keys are few (spans spread one row's keys over the GPU)
    const uint64_t ctas = (uint64_t)a.ns * a.groups * ((a.group_queries() + KT - 1) / KT);
    return a.group_queries() >= KT && (ctas * 8 >= sms || a.max_pos <= 2048);
}

int qb_launch_shared_kv_prefill(qb_ctx *ctx, const QbSharedKv &a) {
    const QbLatent &L = a.at;
    const uint32_t NU = units_of(L), stages = pf_smem(NU, 2).total <= SMEM_LIMIT ? 2 : 1, smem = pf_smem(NU, stages).total;
    QB_CUDA(cudaFuncSetAttribute(shared_kv_prefill_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    CUtensorMap map;
    {
        std::lock_guard<std::mutex> lock(g_lock);
        if (g_maps.size() > 4096) g_maps.clear();
        const uint32_t cols = L.groups * L.pitch();
        const MapKey key{ctx->device, L.cache, L.slots, cols};
        auto it = g_maps.find(key);
        if (it == g_maps.end()) {
            CUtensorMap m;
            // a box: one 128-byte column of a 16-key page; columns past a vector read as the next head's (their queries are zero,
            // their outputs not kept), past the last as zero
            QB_TRY(qb_make_tmap_2d(&m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, L.cache, cols, L.slots, (uint64_t)cols * 2, 64, 16, CU_TENSOR_MAP_SWIZZLE_128B));
            it = g_maps.emplace(key, m).first;
        }
        map = it->second;
    }
    QB_CUDA(qb_launch_pdl(ctx->stream, shared_kv_prefill_kernel, dim3(L.ns * L.groups, (L.group_queries() + KT - 1) / KT), dim3(THREADS), (size_t)smem, a, map, NU, stages));
    QB_LAUNCHED(ctx, "shared_kv_prefill_kernel");
    return QB_OK;
}
