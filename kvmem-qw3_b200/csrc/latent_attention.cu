// Latent attention: the cache holds one normalised latent and one rotated key part per token (paged); keys and values of
// every head are linear maps of the latent.  A learned number per head joins the softmax denominator (a sink without key
// or value).
//
// Few rows per sequence (decode), and every row in fp32: the absorbed form.  q_n . (W_uk c) = (W_uk^T q_n) . c, so the key
// projection is applied to the query once (latent_absorb_kernel), all heads of all rows of a sequence then attend the same
// cached vectors over spans of keys (latent_split_tc_kernel, latent_attention_tc.cu; shapes it does not take:
// latent_split_kernel, 16 or 32 (row, head) queries per CTA on mma.sync, the tile of latents serving as keys and as values;
// latent_split_simt_kernel: the same in fp32), and latent_merge_kernel folds the spans, adds the sink and applies W_uv head by head.
//
// Prompt chunks in bfloat16: the latents of all keys are gathered from their pages, expanded to keys and values by one
// GEMM, and latent_prefill_kernel runs a tiled attention per head (128 or 64 rows per CTA, running maximum and sum).
//
// Scores, weights and their sums are fp32; weights enter the value product as bfloat16.
#include "layered.h"
#include "mma_common.cuh"

namespace {
using namespace qbmma;

constexpr int LT = 256;
constexpr float LOG2E = 1.4426950408889634f;

// ---- new rows: rotate the query, normalise the latent, append to the paged cache ----------------------------------------
// grid (rows, 1 + head groups): block y = 0 takes the latent and the shared key part, y > 0 `hpb` query heads.
template <typename T>
__global__ void __launch_bounds__(LT)
latent_prepare_kernel(QbLatent a, uint32_t hpb) {
    QB_PDL_ENTER();
    extern __shared__ float sm[];
    __shared__ float red[LT / 32];
    const uint32_t m = blockIdx.x, s = m / a.R, tid = threadIdx.x, half = a.rot.dims / 2;
    float *cs = sm, *sn = cs + half, *lat = sn + half;
    const int pos = a.seq_pos[s] + (int)(m % a.R);
    const size_t base = (size_t)m * a.stride, ps = (size_t)a.ns * a.R * a.stride;
    const uint32_t hq = a.dim + a.rot_dim, c0 = a.H * hq, k0 = c0 + a.rank;
    for (uint32_t i = tid; i < half; i += LT) qb_rot_angle(a.rot, pos, i, cs[i], sn[i]);
    auto rotated = [&](uint32_t at, uint32_t j) -> float {          // element j of the rotated vector that starts at column `at`
        const float v = qb_sum8(a.proj, base + at + j, a.S, ps);
        if (j >= a.rot.dims) return v;
        uint32_t i, p; bool first;
        qb_rot_pair(a.rot, j, i, p, first);
        const float w = qb_sum8(a.proj, base + at + p, a.S, ps);
        return first ? v * cs[i] - w * sn[i] : v * cs[i] + w * sn[i];
    };
    if (blockIdx.y > 0) {
        __syncthreads();
        const uint32_t h0 = (blockIdx.y - 1) * hpb, nh = min(hpb, a.H - h0);
        const uint32_t dp = a.dimp(), per = dp + a.rotp();
        T *q = (T *)a.q + ((size_t)m * a.H + h0) * per;
#pragma unroll 4
        for (uint32_t i = tid; i < nh * per; i += LT) {
            const uint32_t h = h0 + i / per, e = i % per;
            float v = 0.0f;
            if (e < a.dim) v = qb_sum8(a.proj, base + h * hq + e, a.S, ps);
            else if (e >= dp && e - dp < a.rot_dim) v = rotated(h * hq + a.dim, e - dp);
            q[i] = qb_cast<T>(v);
        }
        return;
    }
    float ss = 0.0f;
    for (uint32_t i = tid; i < a.rank; i += LT) {
        const float v = qb_sum8(a.proj, base + c0 + i, a.S, ps);
        lat[i] = v;
        ss += v * v;
    }
    const float inv = rsqrtf(qb_block_sum(ss, red, LT / 32) / (float)a.rank + a.eps);
    const int64_t at = qb_latent_slot(a, a.page_table + (size_t)s * a.pt_stride, (uint32_t)pos);
    if (at < 0) {
        if (tid == 0) atomicExch(a.err_flag, 3002);                    // an unassigned page: nothing is appended
        return;
    }
    T *slot = (T *)a.cache + (size_t)at * a.pitch();
    const uint32_t rp = a.rankp();
    for (uint32_t i = tid; i < a.pitch(); i += LT) {
        float v = 0.0f;
        if (i < a.rank) v = lat[i] * inv * a.norm_w[i];
        else if (i >= rp && i - rp < a.rot_dim) v = rotated(k0, i - rp);
        slot[i] = qb_cast<T>(v);
    }
}

// ---- absorbed query: qa[row][h] = [W_uk(h)^T q_n | q_r] --------------------------------------------------------------------
// A CTA takes one head, 128 latent columns and AB_ROWS rows; its weights are requested into L2 before it waits for the query.
template <typename T, int AB_ROWS>
__global__ void __launch_bounds__(128)
latent_absorb_kernel(QbLatent a, const uint8_t *__restrict__ rec, uint32_t kc, uint32_t rows) {
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    for (uint32_t i = threadIdx.x; i < 2 * a.dim; i += 128)           // two 128-byte lines per weight row
        if (blockIdx.y * 2 + (i & 1) < kc)
            asm volatile("prefetch.global.L2 [%0];" ::"l"(rec + qb_dense_offset(kc, blockIdx.x * (a.dimp() + a.vdimp()) + (i >> 1), (blockIdx.y * 2 + (i & 1)) * 8)));
    asm volatile("griddepcontrol.wait;" ::: "memory");
    extern __shared__ float sm[];
    const uint32_t h = blockIdx.x, row0 = blockIdx.z * AB_ROWS, tid = threadIdx.x;
    const uint32_t nr = min((uint32_t)AB_ROWS, rows - row0);
    const uint32_t dp = a.dimp(), per = dp + a.rotp(), rp = a.rankp(), pitch = a.pitch();
    float *qs = sm, *red = sm + AB_ROWS * a.dim;                     // red [8 groups][AB_ROWS][128]
    const T *q = (const T *)a.q;
    for (uint32_t i = tid; i < AB_ROWS * a.dim; i += 128) {
        const uint32_t r = i / a.dim, d = i % a.dim;
        qs[i] = r < nr ? qb_f32(q[((size_t)(row0 + r) * a.H + h) * per + d]) : 0.0f;
    }
    __syncthreads();
    const uint32_t cg = tid & 15, dg = tid >> 4, c8 = blockIdx.y * 16 + cg;
    float acc[AB_ROWS][8] = {};
    if (c8 < kc * 8) {
        const uint32_t wr0 = h * (dp + a.vdimp());
#pragma unroll(AB_ROWS == 1 ? 8 : 4)
        for (uint32_t d = dg; d < a.dim; d += 8) {
            const uint4 raw = *reinterpret_cast<const uint4 *>(rec + qb_dense_offset(kc, wr0 + d, c8));
            const __nv_bfloat162 *b = reinterpret_cast<const __nv_bfloat162 *>(&raw);
            float w[8];
#pragma unroll
            for (int i = 0; i < 4; ++i) { const float2 f = __bfloat1622float2(b[i]); w[2 * i] = f.x; w[2 * i + 1] = f.y; }
#pragma unroll
            for (int r = 0; r < AB_ROWS; ++r) {
                const float qv = qs[r * a.dim + d];
#pragma unroll
                for (int i = 0; i < 8; ++i) acc[r][i] = fmaf(qv, w[i], acc[r][i]);
            }
        }
    }
#pragma unroll
    for (int r = 0; r < AB_ROWS; ++r)
#pragma unroll
        for (int i = 0; i < 8; ++i) red[(dg * AB_ROWS + r) * 128 + cg * 8 + i] = acc[r][i];
    __syncthreads();
    T *qa = (T *)a.qa;
    const uint32_t col = blockIdx.y * 128 + tid;
    for (uint32_t r = 0; r < nr; ++r) {
        float v = 0.0f;
#pragma unroll
        for (int g = 0; g < 8; ++g) v += red[(g * AB_ROWS + r) * 128 + tid];
        T *dst = qa + ((size_t)(row0 + r) * a.H + h) * pitch;
        if (col < rp) dst[col] = qb_cast<T>(col < a.rank ? v : 0.0f);
        if (blockIdx.y == 0)
            for (uint32_t j = tid; j < a.rotp(); j += 128) dst[rp + j] = q[((size_t)(row0 + r) * a.H + h) * per + dp + j];
    }
}

// ---- absorbed attention, fp32 arithmetic: 8 (row, head) queries per CTA, a warp each for the scores ------------------------
constexpr int SQ = 8, SK = 32, SCOLS = 4;                             // value columns per thread: up to 4 x 256
template <typename T>
__global__ void __launch_bounds__(LT)
latent_split_simt_kernel(QbLatent a, uint32_t n_splits) {
    QB_PDL_ENTER();
    extern __shared__ float sm[];
    const uint32_t D = a.pitch(), DP = D + 1, tid = threadIdx.x, w = tid >> 5, lane = tid & 31;
    float *qs = sm, *ts = qs + SQ * D, *pr = ts + SK * DP, *al = pr + SQ * SK;
    const uint32_t split = blockIdx.x, sg = blockIdx.z, s = sg / a.groups, grp = sg % a.groups, hg = a.heads_per_group(), nq = a.R * hg, q0 = blockIdx.y * SQ;
    const int base = a.seq_pos[s];
    const uint32_t span = qb_latent_span((uint32_t)base + a.R, a.max_splits);
    const uint32_t q_last = min(q0 + SQ, nq) - 1;
    const int k_begin = (int)(split * span), k_end = min(k_begin + (int)span, base + (int)(q_last / hg) + 1);
    if (k_begin >= k_end) return;
    const T *qa = (const T *)a.qa + ((size_t)sg * nq + q0) * D;
    for (uint32_t i = tid; i < SQ * D; i += LT) qs[i] = q0 + i / D < nq ? qb_f32(qa[i]) : 0.0f;
    const int my_pos = q0 + w < nq ? base + (int)((q0 + w) / hg) : -1;
    const int32_t *pt = a.page_table + (size_t)s * a.pt_stride;
    float mx = -INFINITY, sum = 0.0f, acc[SQ][SCOLS] = {};
    for (int kt = k_begin; kt < k_end; kt += SK) {
        __syncthreads();
        for (uint32_t i = tid; i < SK * D; i += LT) {
            const uint32_t j = i / D, e = i % D;
            const int key = kt + (int)j;
            float v = 0.0f;
            const int64_t at = key < k_end ? qb_latent_slot(a, pt, (uint32_t)key) : -1;
            if (at >= 0) v = qb_f32(((const T *)a.cache)[((size_t)at * a.groups + grp) * D + e]);
            ts[j * DP + e] = v;
        }
        __syncthreads();
        float sc = 0.0f;
        for (uint32_t e = 0; e < D; ++e) sc = fmaf(qs[w * D + e], ts[lane * DP + e], sc);
        const int key = kt + (int)lane;
        if (a.key_scale && key < k_end) {
            const int64_t at = qb_latent_slot(a, pt, (uint32_t)key);
            sc *= at >= 0 ? a.key_scale[(size_t)at * a.groups + grp] : 0.0f;
        }
        sc = key <= my_pos && key < k_end ? sc * a.scale : -INFINITY;
        const float nm = fmaxf(mx, warp_max(sc));
        const float p = sc == -INFINITY ? 0.0f : expf(sc - nm), alpha = mx == -INFINITY ? 0.0f : expf(mx - nm);
        sum = sum * alpha + warp_sum(p);
        mx = nm;
        pr[w * SK + lane] = p;
        if (lane == 0) al[w] = alpha;
        __syncthreads();
#pragma unroll
        for (int i = 0; i < SCOLS; ++i) {
            const uint32_t c = tid + i * LT;
            if (c < a.rank) {
#pragma unroll
                for (int q = 0; q < SQ; ++q) acc[q][i] *= al[q];
                for (int j = 0; j < SK; ++j) {
                    const float v = ts[j * DP + c];
#pragma unroll
                    for (int q = 0; q < SQ; ++q) acc[q][i] = fmaf(pr[q * SK + j], v, acc[q][i]);
                }
            }
        }
    }
    if (lane == 0 && q0 + w < nq) {
        float *ml = a.part_ml + (((size_t)sg * nq + q0 + w) * n_splits + split) * 2;
        ml[0] = mx;
        ml[1] = sum;
    }
#pragma unroll
    for (int q = 0; q < SQ; ++q)
        if (q0 + q < nq) {
            float *dst = a.part_acc + (((size_t)sg * nq + q0 + q) * n_splits + split) * a.rank;
#pragma unroll
            for (int i = 0; i < SCOLS; ++i) if (tid + i * LT < a.rank) dst[tid + i * LT] = acc[q][i];
        }
}

// ---- mma.sync pieces ----------------------------------------------------------------------------------------------------------
// ---- the two per-head products for many rows (batched decode, bfloat16): 32 rows x 64 columns per CTA on mma.sync -------------
// A warp takes 8 columns.  The weights are requested before the CTA waits for the kernel in front of it.
constexpr uint32_t PR = 32, PC = 64;

// qa[row][h] = [W_uk(h)^T q_n | q_r]: grid (H, latent columns / 64, rows / 32)
__global__ void __launch_bounds__(LT)
latent_absorb_mma_kernel(QbLatent a, const uint8_t *__restrict__ rec, uint32_t kc, uint32_t rows) {
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    extern __shared__ __align__(16) uint8_t smem[];
    const uint32_t h = blockIdx.x, c0 = blockIdx.y * PC, r0 = blockIdx.z * PR, tid = threadIdx.x, w = tid >> 5, lane = tid & 31;
    const uint32_t dp = a.dimp(), per = dp + a.rotp(), rp = a.rankp(), D = a.pitch(), qp = (dp + 8) * 2, wp = (PC + 8) * 2;
    const uint32_t qs = s32(smem), ws = qs + PR * qp;
    for (uint32_t i = tid; i < dp * 8; i += LT)                         // [dp rows][64 columns]
        cp16(ws + (i >> 3) * wp + (i & 7) * 16, rec + qb_dense_offset(kc, h * (dp + a.vdimp()) + (i >> 3), blockIdx.y * 8 + (i & 7)), true);
    cp_commit();
    asm volatile("griddepcontrol.wait;" ::: "memory");
    const __nv_bfloat16 *q = (const __nv_bfloat16 *)a.q;
    for (uint32_t i = tid; i < PR * (dp / 8); i += LT) {
        const uint32_t r = i / (dp / 8), c = i % (dp / 8);
        const bool ok = r0 + r < rows;
        cp16(qs + r * qp + c * 16, ok ? q + ((size_t)(r0 + r) * a.H + h) * per + c * 8 : q, ok);
    }
    cp_commit();
    cp_wait<0>();
    __syncthreads();
    float acc[2][4] = {};
    for (uint32_t k = 0; k < dp / 16; ++k) {
        uint32_t b[2];
        ldsm2t(b, ws + (k * 16 + (lane & 15)) * wp + w * 16);
#pragma unroll
        for (int t = 0; t < 2; ++t) {
            uint32_t f[4];
            ldsm4(f, qs + (t * 16 + (lane & 15)) * qp + k * 32 + (lane >> 4) * 16);
            mma(acc[t], f, b[0], b[1]);
        }
    }
    __nv_bfloat16 *qa = (__nv_bfloat16 *)a.qa;
#pragma unroll
    for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int i = 0; i < 4; i += 2) {
            const uint32_t r = r0 + t * 16 + (lane >> 2) + (i >> 1) * 8, c = c0 + w * 8 + (lane & 3) * 2;
            if (r < rows && c < rp)                                     // (weights past the latent are zero)
                *reinterpret_cast<uint32_t *>(qa + ((size_t)r * a.H + h) * D + c) = pack_bf16(acc[t][i], acc[t][i + 1]);
        }
    if (blockIdx.y == 0)
        for (uint32_t i = tid; i < PR * a.rotp(); i += LT) {
            const uint32_t r = r0 + i / a.rotp(), j = i % a.rotp();
            if (r < rows) qa[((size_t)r * a.H + h) * D + rp + j] = q[((size_t)r * a.H + h) * per + dp + j];
        }
}

// Folds the spans, adds the sink, applies W_uv: grid (H, rows / 32, value dimensions / 64)
__global__ void __launch_bounds__(LT)
latent_merge_mma_kernel(QbLatent a, const uint8_t *__restrict__ rec, uint32_t kc, uint32_t rows, uint32_t n_splits) {
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    extern __shared__ __align__(16) uint8_t smem[];
    const uint32_t h = blockIdx.x, r0 = blockIdx.y * PR, v0 = blockIdx.z * PC, tid = threadIdx.x, w = tid >> 5, lane = tid & 31;
    const uint32_t pitch = (kc * 64 + 8) * 2, vp = a.vdimp();
    const uint32_t ls = s32(smem), ws = ls + PR * pitch;
    float *wt = reinterpret_cast<float *>(smem + (PR + PC) * pitch);    // [32][n_splits]
    __shared__ uint32_t cnt[PR];
    for (uint32_t i = tid; i < PC * kc * 8; i += LT) {                  // [64 value rows][latent]
        const uint32_t v = i / (kc * 8), c = i % (kc * 8);
        const bool ok = v0 + v < vp;
        cp16(ws + v * pitch + c * 16, rec + qb_dense_offset(kc, h * (a.dimp() + vp) + a.dimp() + (ok ? v0 + v : 0), c), ok);
    }
    cp_commit();
    asm volatile("griddepcontrol.wait;" ::: "memory");
    for (uint32_t j = w; j < PR; j += LT / 32) {
        const uint32_t m = r0 + j;
        uint32_t n = 0;
        if (m < rows) {
            const uint32_t base = (uint32_t)a.seq_pos[m / a.R], pos = base + m % a.R;
            n = min(pos / qb_latent_span(base + a.R, a.max_splits) + 1, n_splits);
            const float *ml = a.part_ml + ((size_t)m * a.H + h) * n_splits * 2;
            const float sink = a.sink[h];
            float mx = sink;
            for (uint32_t i = lane; i < n; i += 32) mx = fmaxf(mx, ml[2 * i]);
            mx = warp_max(mx);
            float den = 0.0f;
            for (uint32_t i = lane; i < n; i += 32) den += ml[2 * i + 1] * expf(ml[2 * i] - mx);
            den = warp_sum(den) + expf(sink - mx);
            for (uint32_t i = lane; i < n; i += 32) wt[j * n_splits + i] = expf(ml[2 * i] - mx) / den;
        }
        if (lane == 0) cnt[j] = n;
    }
    __syncthreads();
    const uint32_t half = kc * 32;                                      // column pairs
#pragma unroll 4
    for (uint32_t t = tid; t < PR * half; t += LT) {
        const uint32_t r = t / half, c = (t % half) * 2, n = cnt[r];
        const float *acc = a.part_acc + ((size_t)(r0 + r) * a.H + h) * n_splits * a.rank + c;
        float x = 0.0f, y = 0.0f;
        for (uint32_t i = 0; i < n; ++i) {
            const float f = wt[r * n_splits + i];
            if (c < a.rank) x = fmaf(f, acc[(size_t)i * a.rank], x);
            if (c + 1 < a.rank) y = fmaf(f, acc[(size_t)i * a.rank + 1], y);
        }
        *reinterpret_cast<uint32_t *>(smem + r * pitch + c * 2) = pack_bf16(x, y);
    }
    cp_wait<0>();
    __syncthreads();
    float acc[2][4] = {};
    for (uint32_t k = 0; k < kc * 4; ++k) {
        uint32_t b[2];
        ldsm2(b, ws + (w * 8 + (lane & 7)) * pitch + k * 32 + ((lane >> 3) & 1) * 16);
#pragma unroll
        for (int t = 0; t < 2; ++t) {
            uint32_t f[4];
            ldsm4(f, ls + (t * 16 + (lane & 15)) * pitch + k * 32 + (lane >> 4) * 16);
            mma(acc[t], f, b[0], b[1]);
        }
    }
#pragma unroll
    for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const uint32_t r = r0 + t * 16 + (lane >> 2) + (i >> 1) * 8, v = v0 + w * 8 + (lane & 3) * 2 + (i & 1);
            if (r < rows && v < a.vdim) ((__nv_bfloat16 *)a.out.p + (size_t)r * a.out.ld + h * a.vdim)[v] = __float2bfloat16(acc[t][i]);
        }
}

// ---- absorbed attention on mma.sync: 16 MT queries per CTA over one span of keys, 64-key tiles --------------------------------
// 8 warps: for the scores a warp takes 8 of a tile's keys, for the softmax 2 MT queries, for the value product NV x 8 of
// the latent's columns.
constexpr int DKT = 64;
struct SplitSmem {
    uint32_t q, tile, s, p, misc, total;
};
__host__ __device__ inline SplitSmem split_smem(uint32_t D, uint32_t MT) {
    SplitSmem m;
    const uint32_t row = (D + 8) * 2;
    m.q = 0;
    m.tile = m.q + 16 * MT * row;
    m.s = m.tile + 2 * DKT * row;
    m.p = m.s + 16 * MT * 68 * 4;
    m.misc = m.p + 16 * MT * 72 * 2;
    m.total = m.misc + 16 * MT * 4 * 2;
    return m;
}
template <int MT, int NV>
__global__ void __launch_bounds__(LT)
latent_split_kernel(QbLatent a, uint32_t n_splits) {
    QB_PDL_ENTER();
    extern __shared__ __align__(16) uint8_t smem[];
    const uint32_t D = a.pitch(), pitch = (D + 8) * 2, tid = threadIdx.x, w = tid >> 5, lane = tid & 31;
    const SplitSmem L = split_smem(D, MT);
    float *ssm = reinterpret_cast<float *>(smem + L.s), *al = reinterpret_cast<float *>(smem + L.misc);
    __nv_bfloat16 *psm = reinterpret_cast<__nv_bfloat16 *>(smem + L.p);
    const uint32_t split = blockIdx.x, s = blockIdx.z, nq = a.R * a.H, q0 = blockIdx.y * 16 * MT;
    const int base = a.seq_pos[s];
    const uint32_t span = qb_latent_span((uint32_t)base + a.R, a.max_splits);
    const uint32_t q_last = min(q0 + 16 * MT, nq) - 1;
    const int k_begin = (int)(split * span), k_end = min(k_begin + (int)span, base + (int)(q_last / a.H) + 1);
    if (k_begin >= k_end) return;
    const int32_t *pt = a.page_table + (size_t)s * a.pt_stride;
    const __nv_bfloat16 *cache = (const __nv_bfloat16 *)a.cache;
    auto load_tile = [&](int kt, uint32_t st) {
        const uint32_t dst = s32(smem + L.tile) + st * DKT * pitch;
        for (uint32_t i = tid; i < DKT * (D / 8); i += LT) {
            const uint32_t j = i / (D / 8), c = i % (D / 8);
            const int key = kt + (int)j;
            const int64_t at = key < k_end ? qb_latent_slot(a, pt, (uint32_t)key) : -1;
            cp16(dst + j * pitch + c * 16, at >= 0 ? cache + (size_t)at * D + c * 8 : cache, at >= 0);
        }
        cp_commit();
    };
    {
        const __nv_bfloat16 *qa = (const __nv_bfloat16 *)a.qa + ((size_t)s * nq + q0) * D;
        for (uint32_t i = tid; i < 16 * MT * (D / 8); i += LT) {
            const uint32_t j = i / (D / 8), c = i % (D / 8);
            const bool ok = q0 + j < nq;
            cp16(s32(smem + L.q) + j * pitch + c * 16, ok ? qa + (size_t)j * D + c * 8 : qa, ok);
        }
    }
    load_tile(k_begin, 0);
    float o[MT][NV][4];
#pragma unroll
    for (int t = 0; t < MT; ++t)
#pragma unroll
        for (int n = 0; n < NV; ++n)
#pragma unroll
            for (int i = 0; i < 4; ++i) o[t][n][i] = 0.0f;
    float mx[2 * MT], sum[2 * MT];
    int qpos[2 * MT];
#pragma unroll
    for (int i = 0; i < 2 * MT; ++i) {
        const uint32_t q = q0 + w * 2 * MT + i;
        mx[i] = -INFINITY; sum[i] = 0.0f;
        qpos[i] = q < nq ? base + (int)(q / a.H) : -1;
    }
    const uint32_t rankp = a.rankp();
    uint32_t it = 0;
    for (int kt = k_begin; kt < k_end; kt += DKT, ++it) {
        const uint32_t st = it & 1;
        if (kt + DKT < k_end) { load_tile(kt + DKT, st ^ 1); cp_wait<1>(); }
        else cp_wait<0>();
        __syncthreads();
        const uint32_t tile = s32(smem + L.tile) + st * DKT * pitch;
        {   // scores: queries x the warp's 8 keys
            float sc[MT][4] = {};
            const uint32_t baddr = tile + (w * 8 + (lane & 7)) * pitch + ((lane >> 3) & 1) * 16;
            const uint32_t aaddr = s32(smem + L.q) + (lane & 15) * pitch + (lane >> 4) * 16;
            for (uint32_t k = 0; k < D / 16; ++k) {
                uint32_t b[2];
                ldsm2(b, baddr + k * 32);
#pragma unroll
                for (int t = 0; t < MT; ++t) {
                    uint32_t q[4];
                    ldsm4(q, aaddr + t * 16 * pitch + k * 32);
                    mma(sc[t], q, b[0], b[1]);
                }
            }
            const uint32_t r = lane >> 2, c = w * 8 + (lane & 3) * 2;
#pragma unroll
            for (int t = 0; t < MT; ++t) {
                ssm[(t * 16 + r) * 68 + c] = sc[t][0]; ssm[(t * 16 + r) * 68 + c + 1] = sc[t][1];
                ssm[(t * 16 + r + 8) * 68 + c] = sc[t][2]; ssm[(t * 16 + r + 8) * 68 + c + 1] = sc[t][3];
            }
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 2 * MT; ++i) {
            const uint32_t q = w * 2 * MT + i;
            const int key = kt + (int)lane;
            const float s0 = key <= qpos[i] && key < k_end ? ssm[q * 68 + lane] * a.scale : -INFINITY;
            const float s1 = key + 32 <= qpos[i] && key + 32 < k_end ? ssm[q * 68 + lane + 32] * a.scale : -INFINITY;
            const float nm = fmaxf(mx[i], warp_max(fmaxf(s0, s1)));
            const float ref = nm == -INFINITY ? 0.0f : nm;
            const float p0 = exp2f((s0 - ref) * LOG2E), p1 = exp2f((s1 - ref) * LOG2E);
            const float alpha = exp2f((mx[i] - ref) * LOG2E);
            sum[i] = sum[i] * alpha + warp_sum(p0 + p1);
            mx[i] = nm;
            psm[q * 72 + lane] = __float2bfloat16(p0);
            psm[q * 72 + lane + 32] = __float2bfloat16(p1);
            if (lane == 0) al[q] = alpha;
        }
        __syncthreads();
#pragma unroll
        for (int t = 0; t < MT; ++t) {
            const float a0 = al[t * 16 + (lane >> 2)], a1 = al[t * 16 + (lane >> 2) + 8];
#pragma unroll
            for (int n = 0; n < NV; ++n) { o[t][n][0] *= a0; o[t][n][1] *= a0; o[t][n][2] *= a1; o[t][n][3] *= a1; }
        }
#pragma unroll
        for (int k = 0; k < DKT / 16; ++k) {
            uint32_t p[MT][4];
#pragma unroll
            for (int t = 0; t < MT; ++t) ldsm4(p[t], s32(psm) + (t * 16 + (lane & 15)) * 144 + k * 32 + (lane >> 4) * 16);
#pragma unroll
            for (int n = 0; n < NV; n += 2) {
                const uint32_t col = (w * NV + n) * 8;
                if (col >= rankp) break;                               // uniform over the warp; rankp is a multiple of 16
                uint32_t b[4];
                ldsm4t(b, tile + (k * 16 + (lane & 15)) * pitch + (col + (lane >> 4) * 8) * 2);
#pragma unroll
                for (int t = 0; t < MT; ++t) { mma(o[t][n], p[t], b[0], b[1]); mma(o[t][n + 1], p[t], b[2], b[3]); }
            }
        }
        __syncthreads();                                               // the tile may be overwritten
    }
#pragma unroll
    for (int i = 0; i < 2 * MT; ++i) {
        const uint32_t q = q0 + w * 2 * MT + i;
        if (lane == 0 && q < nq) {
            float *ml = a.part_ml + (((size_t)s * nq + q) * n_splits + split) * 2;
            ml[0] = mx[i];
            ml[1] = sum[i];
        }
    }
#pragma unroll
    for (int t = 0; t < MT; ++t)
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            const uint32_t col = (w * NV + n) * 8 + (lane & 3) * 2;
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const uint32_t q = q0 + t * 16 + (lane >> 2) + (i >> 1) * 8, c = col + (i & 1);
                if (q < nq && c < a.rank) a.part_acc[(((size_t)s * nq + q) * n_splits + split) * a.rank + c] = o[t][n][i];
            }
        }
}

// ---- fold the spans, add the sink, apply W_uv: grid (H, rows / MB, slices of the value dimensions) ----------------------------
template <typename T, int MB>
__global__ void __launch_bounds__(LT)
latent_merge_kernel(QbLatent a, const uint8_t *__restrict__ rec, uint32_t kc, uint32_t rows, uint32_t n_splits) {
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    extern __shared__ float sm[];
    const uint32_t h = blockIdx.x, m0 = blockIdx.y * MB, tid = threadIdx.x, w = tid >> 5, lane = tid & 31;
    const uint32_t per = (a.vdim + gridDim.z - 1) / gridDim.z, v0 = blockIdx.z * per, v1 = min(a.vdim, v0 + per);
    const uint32_t wr0 = h * (a.dimp() + a.vdimp()) + a.dimp();
    for (uint32_t i = tid; v0 < v1 && i < (v1 - v0) * kc; i += LT)     // this CTA's weights, into L2 while the spans are still computed
        asm volatile("prefetch.global.L2 [%0];" ::"l"(rec + qb_dense_offset(kc, wr0 + v0 + i / kc, (i % kc) * 8)));
    asm volatile("griddepcontrol.wait;" ::: "memory");
    float *wt = sm, *lat = sm + ((MB * n_splits + 3) & ~3u);            // weights of the spans, the merged latents [MB][kc * 64]
    __shared__ uint32_t cnt[MB];
    if (w < MB) {
        const uint32_t m = m0 + w;
        uint32_t n = 0;
        if (m < rows) {
            const uint32_t base = (uint32_t)a.seq_pos[m / a.R], pos = base + m % a.R;
            n = min(pos / qb_latent_span(base + a.R, a.max_splits) + 1, n_splits);
            const float *ml = a.part_ml + ((size_t)m * a.H + h) * n_splits * 2;
            const float sink = a.sink[h];
            float mx = sink;
            for (uint32_t i = lane; i < n; i += 32) mx = fmaxf(mx, ml[2 * i]);
            mx = warp_max(mx);
            float den = 0.0f;
            for (uint32_t i = lane; i < n; i += 32) den += ml[2 * i + 1] * expf(ml[2 * i] - mx);
            den = warp_sum(den) + expf(sink - mx);
            for (uint32_t i = lane; i < n; i += 32) wt[w * n_splits + i] = expf(ml[2 * i] - mx) / den;
        }
        if (lane == 0) cnt[w] = n;
    }
    __syncthreads();
#pragma unroll 2
    for (uint32_t t = tid; t < MB * kc * 64; t += LT) {
        const uint32_t r = t / (kc * 64), c = t % (kc * 64), n = cnt[r];
        float v = 0.0f;
        if (c < a.rank) {
            const float *acc = a.part_acc + ((size_t)(m0 + r) * a.H + h) * n_splits * a.rank + c;
#pragma unroll 8
            for (uint32_t i = 0; i < n; ++i) v = fmaf(wt[r * n_splits + i], acc[(size_t)i * a.rank], v);
        }
        lat[t] = v;
    }
    __syncthreads();
    // four value dimensions per warp at a time: their weights are in flight together and share the reads of the latents
    constexpr int NVW = 4;
    for (uint32_t v = v0 + w * NVW; v < v1; v += LT / 32 * NVW) {
        float acc[NVW][MB] = {};
        for (uint32_t c8 = lane; c8 < kc * 8; c8 += 32) {
            uint4 raw[NVW];
#pragma unroll
            for (int j = 0; j < NVW; ++j) raw[j] = *reinterpret_cast<const uint4 *>(rec + qb_dense_offset(kc, wr0 + min(v + j, v1 - 1), c8));
#pragma unroll
            for (int r = 0; r < MB; ++r) {
                const float4 l0 = *reinterpret_cast<const float4 *>(lat + r * kc * 64 + c8 * 8), l1 = *reinterpret_cast<const float4 *>(lat + r * kc * 64 + c8 * 8 + 4);
#pragma unroll
                for (int j = 0; j < NVW; ++j) {
                    const __nv_bfloat162 *b = reinterpret_cast<const __nv_bfloat162 *>(&raw[j]);
                    const float2 f0 = __bfloat1622float2(b[0]), f1 = __bfloat1622float2(b[1]), f2 = __bfloat1622float2(b[2]), f3 = __bfloat1622float2(b[3]);
                    acc[j][r] = fmaf(f0.x, l0.x, fmaf(f0.y, l0.y, fmaf(f1.x, l0.z, fmaf(f1.y, l0.w, acc[j][r]))));
                    acc[j][r] = fmaf(f2.x, l1.x, fmaf(f2.y, l1.y, fmaf(f3.x, l1.z, fmaf(f3.y, l1.w, acc[j][r]))));
                }
            }
        }
#pragma unroll
        for (int j = 0; j < NVW; ++j)
#pragma unroll
            for (int r = 0; r < MB; ++r) {
                const float t = warp_sum(acc[j][r]);
                if (lane == 0 && v + j < v1 && m0 + r < rows) ((T *)a.out.p + (size_t)(m0 + r) * a.out.ld + h * a.vdim)[v + j] = qb_cast<T>(t);
            }
    }
}

// ---- prompt chunks ---------------------------------------------------------------------------------------------------------------
// The latents and shared key parts of keys [0, n) of a sequence, out of their pages.
__global__ void __launch_bounds__(LT)
latent_gather_kernel(QbLatent a, uint32_t n) {
    QB_PDL_ENTER();
    const uint32_t D8 = a.pitch() / 8, r8 = a.rankp() / 8;
    const uint64_t i = (uint64_t)blockIdx.x * LT + threadIdx.x;
    if (i >= (uint64_t)n * D8) return;
    const uint32_t key = (uint32_t)(i / D8), c = (uint32_t)(i % D8);
    const int64_t at = qb_latent_slot(a, a.page_table, key);
    const uint4 v = at >= 0 ? *reinterpret_cast<const uint4 *>((const __nv_bfloat16 *)a.cache + (size_t)at * a.pitch() + c * 8) : make_uint4(0u, 0u, 0u, 0u);
    if (c < r8) *reinterpret_cast<uint4 *>((__nv_bfloat16 *)a.lat.p + (size_t)key * a.lat.ld + c * 8) = v;
    else *reinterpret_cast<uint4 *>(a.kr + (size_t)key * a.rotp() + (c - r8) * 8) = v;
}

// One head, 16 query rows per warp, 64-key tiles, running maximum and sum.  grid (row blocks, H).
template <int NV>                                                         // value tiles of 8: vdimp <= 8 NV
__global__ void __launch_bounds__(256)
latent_prefill_kernel(QbLatent a) {
    QB_PDL_ENTER();
    extern __shared__ __align__(16) uint8_t smem[];
    const uint32_t tid = threadIdx.x, nt = blockDim.x, w = tid >> 5, lane = tid & 31, nw = nt >> 5;
    const uint32_t dp = a.dimp(), rp = a.rotp(), DK = dp + rp, vp = a.vdimp(), kp = (DK + 8) * 2, vpitch = (vp + 8) * 2;
    const uint32_t h = blockIdx.y, row0 = (gridDim.x - 1 - blockIdx.x) * 16 * nw;          // longest blocks first
    const uint32_t qs = s32(smem), ks = qs + 16 * nw * kp, vs = ks + 2 * 64 * kp;
    const int base = a.seq_pos[0];
    const uint32_t rlast = min(row0 + 16 * nw, a.R) - 1;
    const int k_end = base + (int)rlast + 1;
    const uint32_t ldkv = a.H * (dp + vp);
    const __nv_bfloat16 *kv = a.kv + h * (dp + vp);
    auto load_tile = [&](int kt, uint32_t st) {
        const uint32_t n8 = (DK + vp) / 8;
        for (uint32_t i = tid; i < 64 * n8; i += nt) {
            const uint32_t j = i / n8, c = i % n8;
            const int key = kt + (int)j;
            const bool ok = key < k_end;
            if (c < DK / 8) {
                const __nv_bfloat16 *src = c < dp / 8 ? kv + (size_t)key * ldkv + c * 8 : a.kr + (size_t)key * rp + (c - dp / 8) * 8;
                cp16(ks + (st * 64 + j) * kp + c * 16, ok ? src : a.kv, ok);
            } else {
                cp16(vs + (st * 64 + j) * vpitch + (c - DK / 8) * 16, ok ? kv + (size_t)key * ldkv + dp + (c - DK / 8) * 8 : a.kv, ok);
            }
        }
        cp_commit();
    };
    {
        const __nv_bfloat16 *q = (const __nv_bfloat16 *)a.q;
        for (uint32_t i = tid; i < 16 * nw * (DK / 8); i += nt) {
            const uint32_t j = i / (DK / 8), c = i % (DK / 8);
            const bool ok = row0 + j < a.R;
            cp16(qs + j * kp + c * 16, ok ? q + ((size_t)(row0 + j) * a.H + h) * DK + c * 8 : q, ok);
        }
    }
    load_tile(0, 0);
    float o[NV][4];
#pragma unroll
    for (int n = 0; n < NV; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) o[n][i] = 0.0f;
    float mx[2] = {-INFINITY, -INFINITY}, sum[2] = {0.0f, 0.0f};
    const int pr[2] = {base + (int)(row0 + w * 16 + (lane >> 2)), base + (int)(row0 + w * 16 + (lane >> 2)) + 8};
    const int warp_last = base + (int)(row0 + w * 16 + 15);
    const float sl = a.scale * LOG2E;
    uint32_t it = 0;
    for (int kt = 0; kt < k_end; kt += 64, ++it) {
        const uint32_t st = it & 1;
        if (kt + 64 < k_end) { load_tile(kt + 64, st ^ 1); cp_wait<1>(); }
        else cp_wait<0>();
        __syncthreads();
        if (kt <= warp_last) {                                            // some key of the tile is visible to the warp
            float sc[8][4] = {};
            const uint32_t aaddr = qs + (w * 16 + (lane & 15)) * kp + (lane >> 4) * 16;
            const uint32_t baddr = ks + (st * 64 + (lane >> 4) * 8 + (lane & 7)) * kp + ((lane >> 3) & 1) * 16;
            for (uint32_t k = 0; k < DK / 16; ++k) {
                uint32_t q[4];
                ldsm4(q, aaddr + k * 32);
#pragma unroll
                for (int n = 0; n < 8; n += 2) {
                    uint32_t b[4];
                    ldsm4(b, baddr + n * 8 * kp + k * 32);
                    mma(sc[n], q, b[0], b[1]);
                    mma(sc[n + 1], q, b[2], b[3]);
                }
            }
            const bool edge = kt + 63 > base + (int)(row0 + w * 16);      // the diagonal crosses the tile
            float tm[2] = {-INFINITY, -INFINITY};
#pragma unroll
            for (int n = 0; n < 8; ++n)
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    float v = sc[n][i] * sl;
                    if (edge && kt + n * 8 + (int)(lane & 3) * 2 + (i & 1) > pr[i >> 1]) v = -INFINITY;
                    sc[n][i] = v;
                    tm[i >> 1] = fmaxf(tm[i >> 1], v);
                }
            float alpha[2], ref[2];
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                tm[i] = fmaxf(tm[i], __shfl_xor_sync(0xffffffffu, tm[i], 1));
                tm[i] = fmaxf(tm[i], __shfl_xor_sync(0xffffffffu, tm[i], 2));
                const float nm = fmaxf(mx[i], tm[i]);
                ref[i] = nm == -INFINITY ? 0.0f : nm;
                alpha[i] = exp2f(mx[i] - ref[i]);
                mx[i] = nm;
                sum[i] *= alpha[i];
            }
#pragma unroll
            for (int n = 0; n < 8; ++n)
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    sc[n][i] = exp2f(sc[n][i] - ref[i >> 1]);
                    sum[i >> 1] += sc[n][i];
                }
#pragma unroll
            for (int n = 0; n < NV; ++n) { o[n][0] *= alpha[0]; o[n][1] *= alpha[0]; o[n][2] *= alpha[1]; o[n][3] *= alpha[1]; }
            const uint32_t vaddr = vs + (st * 64 + (lane & 15)) * vpitch + (lane >> 4) * 16;
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const uint32_t p[4] = {pack_bf16(sc[2 * k][0], sc[2 * k][1]), pack_bf16(sc[2 * k][2], sc[2 * k][3]),
                                       pack_bf16(sc[2 * k + 1][0], sc[2 * k + 1][1]), pack_bf16(sc[2 * k + 1][2], sc[2 * k + 1][3])};
#pragma unroll
                for (int n = 0; n < NV; n += 2) {
                    if (n * 8 >= (int)vp) break;
                    uint32_t b[4];
                    ldsm4t(b, vaddr + k * 16 * vpitch + n * 16);
                    mma(o[n], p, b[0], b[1]);
                    mma(o[n + 1], p, b[2], b[3]);
                }
            }
        }
        __syncthreads();
    }
    const float sink = a.sink[h] * LOG2E;                                 // scores carry log2(e)
    __nv_bfloat16 *out = (__nv_bfloat16 *)a.out.p;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], 1);
        sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], 2);
        const float m = fmaxf(mx[i], sink);
        const float f = exp2f(mx[i] - m), inv = f / (sum[i] * f + exp2f(sink - m));
        const uint32_t row = row0 + w * 16 + (lane >> 2) + i * 8;
        if (row < a.R)
#pragma unroll
            for (int n = 0; n < NV; ++n)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const uint32_t v = n * 8 + (lane & 3) * 2 + e;
                    if (v < a.vdim) out[(size_t)row * a.out.ld + h * a.vdim + v] = __float2bfloat16(o[n][i * 2 + e] * inv);
                }
    }
}

template <int NV>
int launch_prefill(qb_ctx *ctx, const QbLatent &a) {
    const uint32_t nw = a.R >= 128 && (uint64_t)((a.R + 127) / 128) * a.H >= 96 ? 8 : 4;
    const uint32_t kp = (a.dimp() + a.rotp() + 8) * 2, vp = (a.vdimp() + 8) * 2;
    const size_t smem = (size_t)(16 * nw + 128) * kp + 128 * vp;
    QB_REQUIRE(smem <= 227 * 1024, "latent attention: heads of %u + %u dimensions do not fit", a.dim + a.rot_dim, a.vdim);
    QB_CUDA(cudaFuncSetAttribute(latent_prefill_kernel<NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    QB_CUDA(qb_launch_pdl(ctx->stream, latent_prefill_kernel<NV>, dim3((a.R + 16 * nw - 1) / (16 * nw), a.H), dim3(32 * nw), smem, a));
    QB_LAUNCHED(ctx, "latent_prefill_kernel");
    return QB_OK;
}

template <int MT, int NV>
int launch_split(qb_ctx *ctx, const QbLatent &a, uint32_t n_splits) {
    const size_t smem = split_smem(a.pitch(), MT).total;
    QB_CUDA(cudaFuncSetAttribute(latent_split_kernel<MT, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    QB_CUDA(qb_launch_pdl(ctx->stream, latent_split_kernel<MT, NV>, dim3(n_splits, (a.R * a.H + 16 * MT - 1) / (16 * MT), a.ns), dim3(LT), smem, a, n_splits));
    QB_LAUNCHED(ctx, "latent_split_kernel");
    return QB_OK;
}
template <int MT>
int launch_split_nv(qb_ctx *ctx, const QbLatent &a, uint32_t n_splits) {
    if (a.rankp() <= 128) return launch_split<MT, 2>(ctx, a, n_splits);
    if (a.rankp() <= 256) return launch_split<MT, 4>(ctx, a, n_splits);
    return launch_split<MT, 8>(ctx, a, n_splits);
}
template <typename T>
int launch_simt(qb_ctx *ctx, const QbLatent &a, uint32_t n_splits) {
    const uint32_t D = a.pitch();
    const size_t smem = ((size_t)SQ * D + SK * (D + 1) + SQ * SK + SQ) * sizeof(float);
    QB_REQUIRE(smem <= 227 * 1024 && a.rank <= SCOLS * LT, "latent attention: a latent of %u + %u does not fit", a.rank, a.rot_dim);
    QB_CUDA(cudaFuncSetAttribute(latent_split_simt_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    QB_CUDA(qb_launch_pdl(ctx->stream, latent_split_simt_kernel<T>, dim3(n_splits, (a.group_queries() + SQ - 1) / SQ, a.ns * a.groups), dim3(LT), smem, a, n_splits));
    QB_LAUNCHED(ctx, "latent_split_simt_kernel");
    return QB_OK;
}

template <typename T, int AB>
int launch_absorb(qb_ctx *ctx, const QbLatent &a, uint32_t rows) {
    const size_t smem = ((size_t)AB * a.dim + 8 * AB * 128) * sizeof(float);
    QB_REQUIRE(smem <= 227 * 1024, "latent attention: %u query dimensions do not fit", a.dim);
    QB_CUDA(cudaFuncSetAttribute(latent_absorb_kernel<T, AB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    QB_CUDA(qb_launch_pdl(ctx->stream, latent_absorb_kernel<T, AB>, dim3(a.H, (a.rankp() + 127) / 128, (rows + AB - 1) / AB), dim3(128), smem, a,
                          (const uint8_t *)a.ukv->rec, a.ukv->kc, rows));
    QB_LAUNCHED(ctx, "latent_absorb_kernel");
    return QB_OK;
}
template <typename T, int MB>
int launch_merge(qb_ctx *ctx, const QbLatent &a, uint32_t rows, uint32_t n_splits) {
    const uint32_t kc = a.ukv->kc, groups = (rows + MB - 1) / MB;
    const size_t smem = (((size_t)MB * n_splits + 3) / 4 * 4 + MB * kc * 64) * sizeof(float);
    QB_REQUIRE(smem <= 227 * 1024, "latent attention: a latent of %u does not fit", a.rank);
    QB_CUDA(cudaFuncSetAttribute(latent_merge_kernel<T, MB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    const uint32_t vz = std::max(1u, std::min((a.vdim + 31) / 32, (2u * (uint32_t)ctx->sm_count) / (a.H * groups)));
    QB_CUDA(qb_launch_pdl(ctx->stream, latent_merge_kernel<T, MB>, dim3(a.H, groups, vz), dim3(LT), smem, a, (const uint8_t *)a.ukv->rec, kc, rows, n_splits));
    QB_LAUNCHED(ctx, "latent_merge_kernel");
    return QB_OK;
}

template <typename T>
int latent_absorbed(qb_ctx *ctx, QbLatent a) {
    const uint32_t rows = a.ns * a.R;
    if (a.R > QB_LAT_ABSORB_ROWS) a.max_splits = 1;          // the rows alone fill the GPU
    const uint32_t n_splits = std::min(a.max_splits, (a.max_pos + 63) / 64);
    const size_t sm_ab = (size_t)PR * (a.dimp() + 8) * 2 + (size_t)a.dimp() * (PC + 8) * 2;
    const size_t sm_me = (size_t)(PR + PC) * (a.ukv->kc * 64 + 8) * 2 + (size_t)PR * n_splits * sizeof(float);
    const bool many = !a.f32 && rows >= 8 && sm_ab <= 200 * 1024 && sm_me <= 200 * 1024;
    if (many) {
        QB_CUDA(cudaFuncSetAttribute(latent_absorb_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm_ab));
        QB_CUDA(qb_launch_pdl(ctx->stream, latent_absorb_mma_kernel, dim3(a.H, (a.rankp() + PC - 1) / PC, (rows + PR - 1) / PR), dim3(LT), sm_ab, a,
                              (const uint8_t *)a.ukv->rec, a.ukv->kc, rows));
        QB_LAUNCHED(ctx, "latent_absorb_mma_kernel");
    } else if (rows == 1) QB_TRY((launch_absorb<T, 1>(ctx, a, rows)));
    else QB_TRY((launch_absorb<T, 8>(ctx, a, rows)));
    const uint32_t MT = a.R * a.H > 16 ? 2 : 1;
    static const bool use_tc = qb_env_u32("QW3B200_LATENT_TC", 1) != 0;       // 0: the mma.sync form, for comparison
    if (use_tc && a.R <= QB_LAT_ABSORB_ROWS && qb_latent_tc_supports(a)) {
        QB_TRY(qb_launch_latent_split_tc(ctx, a, n_splits));
    } else if (!a.f32 && a.rankp() <= 512 && split_smem(a.pitch(), MT).total <= 227 * 1024) {
        if (MT == 2) QB_TRY(launch_split_nv<2>(ctx, a, n_splits));
        else QB_TRY(launch_split_nv<1>(ctx, a, n_splits));
    } else {
        QB_TRY(launch_simt<T>(ctx, a, n_splits));
    }
    if (many) {
        QB_CUDA(cudaFuncSetAttribute(latent_merge_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm_me));
        QB_CUDA(qb_launch_pdl(ctx->stream, latent_merge_mma_kernel, dim3(a.H, (rows + PR - 1) / PR, (a.vdimp() + PC - 1) / PC), dim3(LT), sm_me, a,
                              (const uint8_t *)a.ukv->rec, a.ukv->kc, rows, n_splits));
        QB_LAUNCHED(ctx, "latent_merge_mma_kernel");
        return QB_OK;
    }
    if (rows == 1) return launch_merge<T, 1>(ctx, a, rows, n_splits);
    return launch_merge<T, 4>(ctx, a, rows, n_splits);
}

}  // namespace

uint32_t qb_latent_max_splits(const QbLatent &a, uint32_t ns, uint32_t sms) {
    const uint32_t groups = (a.H + 47) / 48;
    return std::max(1u, std::min(64u, sms / (ns * groups)));
}

int qb_launch_latent_split_simt(qb_ctx *ctx, const QbLatent &a, uint32_t n_splits) {
    return a.f32 ? launch_simt<float>(ctx, a, n_splits) : launch_simt<__nv_bfloat16>(ctx, a, n_splits);
}

bool qb_latent_expands(const QbLatent &a) {
    return !a.f32 && a.vdimp() <= 256 && ((size_t)(128 + 128) * (a.dimp() + a.rotp() + 8) + 128 * (a.vdimp() + 8)) * 2 <= 227 * 1024;
}

size_t qb_latent_part_floats(const QbLatent &a, uint32_t rows_cap, uint32_t n_seqs, uint32_t sms) {
    const size_t few = std::max({n_seqs, sms, QB_LAT_ABSORB_ROWS * 64u});       // (sequences x rows each) x spans
    return std::max(few, qb_latent_expands(a) ? (size_t)0 : (size_t)rows_cap) * a.H * a.rank;
}

int qb_launch_latent(qb_ctx *ctx, const QbLatent &args) {
    QbLatent a = args;
    a.err_flag = ctx->err_flag_dev;
    const uint32_t rows = a.ns * a.R;
    QB_REQUIRE(rows > 0 && a.rot.dims <= a.rot_dim && a.rot.dims % 2 == 0 && a.stride == a.H * (a.dim + a.rot_dim) + a.rank + a.rot_dim, "latent attention: bad arguments");
    const size_t sm_p = ((size_t)a.rot.dims + a.rank) * sizeof(float);
    // query heads per CTA: enough elements for its threads, fewer when there are few rows
    const uint32_t per = a.dimp() + a.rotp(), hpb = std::max(1u, (rows <= 64 ? 1024u : 4096u) / per);
    const dim3 grid(rows, 1 + (a.H + hpb - 1) / hpb);
    if (a.f32) QB_CUDA(qb_launch_pdl(ctx->stream, latent_prepare_kernel<float>, grid, dim3(LT), sm_p, a, hpb));
    else QB_CUDA(qb_launch_pdl(ctx->stream, latent_prepare_kernel<__nv_bfloat16>, grid, dim3(LT), sm_p, a, hpb));
    QB_LAUNCHED(ctx, "latent_prepare_kernel");
    if (a.f32) return latent_absorbed<float>(ctx, a);
    if (!a.ingest || a.R <= QB_LAT_ABSORB_ROWS || !qb_latent_expands(a)) return latent_absorbed<__nv_bfloat16>(ctx, a);
    QB_REQUIRE(a.ns == 1 && a.max_pos <= a.lat.cap, "latent attention: %u keys exceed the expansion buffers", a.max_pos);
    const uint64_t n16 = (uint64_t)a.max_pos * (a.pitch() / 8);
    QB_CUDA(qb_launch_pdl(ctx->stream, latent_gather_kernel, dim3((unsigned)((n16 + LT - 1) / LT)), dim3(LT), (size_t)0, a, a.max_pos));
    QB_LAUNCHED(ctx, "latent_gather_kernel");
    QB_TRY(qb_dense_gemm_bf16(ctx, *a.ukv, a.lat, a.max_pos, a.kv, a.ukv->rows));
    if (a.vdimp() <= 64) return launch_prefill<8>(ctx, a);
    if (a.vdimp() <= 128) return launch_prefill<16>(ctx, a);
    return launch_prefill<32>(ctx, a);
}
