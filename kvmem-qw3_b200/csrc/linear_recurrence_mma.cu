// Prompt chunks of the linear recurrences on the tensor cores (bfloat16 models): the block form of linear_recurrence.cu with
// mma.sync.  Every operand -- q, k, v, decayed scores, state -- is the sum of two bfloat16 numbers (16 bits of an fp32 value) and a
// product three of the four terms; sums are fp32, the state stays in fp32 registers from block to block.
//
// A CTA owns 32 value columns of a head and walks the chunk in blocks of 64 rows:
//     P = (Q K^T) . D          4 x 8 tiles of 16 x 8, tiles above the diagonal left out
//     O = diag(a) (Q S) + P V
//     S = keep S + K^T (w V)   a warp owns 16 rows of S (twice 16 for heads over 128)
// The next block's rows are copied to shared memory while this one is computed, where they fit.
#include "linear_recurrence.cuh"
#include "mma_common.cuh"

namespace {
using namespace qbrec;
using namespace qbmma;

constexpr uint32_t RT = 256, VP = VCH + 8, PP = C + 8;       // pitches in elements (16-byte pieces per row: an odd number)

struct MmaSmem { uint32_t qh, ql, kh, kl, vh, vl, wh, wl, ph, pl, sh, sl, pw, nst, raw, total; bool staged; };
__host__ __device__ inline MmaSmem mma_smem(uint32_t dim, uint32_t stage) {
    MmaSmem m;
    const uint32_t DP = (dim + 15) & ~15u, qk = C * (DP + 8) * 2, v = C * VP * 2, p = C * PP * 2, s = DP * VP * 2;
    m.qh = 0; m.ql = m.qh + qk; m.kh = m.ql + qk; m.kl = m.kh + qk;
    m.vh = m.kl + qk; m.vl = m.vh + v; m.wh = m.vl + v; m.wl = m.wh + v;
    m.ph = m.wl + v; m.pl = m.ph + p;
    m.sh = m.pl + p; m.sl = m.sh + s;
    m.pw = m.sl + s; m.nst = m.pw + (C + 4) * 4;
    m.raw = m.nst + DP * 4;
    m.total = m.raw + (stage ? C * (2 * dim + VCH) * 4 : 0);
    return m;
}

// d += (ah + al) (bh + bl) without al bl
__device__ __forceinline__ void mma3(float (&d)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], const uint32_t *bh, const uint32_t *bl) {
    mma(d, ah, bh[0], bh[1]);
    mma(d, ah, bl[0], bl[1]);
    mma(d, al, bh[0], bh[1]);
}

// silu to a few units in the last place of fp32 (the operands keep 16 bits)
__device__ __forceinline__ float silu(float v) { return __fdividef(v, 1.0f + __expf(-v)); }

// grid (value slices, H, sequences); ND: 16-row tiles of the state per warp
template <bool GATED, int ND>
__global__ void __launch_bounds__(RT, 1)
recurrence_mma_kernel(QbRecurrence a, uint32_t staged) {
    QB_PDL_ENTER();
    extern __shared__ __align__(16) uint8_t smem[];
    __shared__ BlockGates bg;
    const MmaSmem L = mma_smem(a.dim, staged);
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y, s = blockIdx.z, v0 = blockIdx.x * VCH;
    const uint32_t nv = min(VCH, a.vdim - v0), DP = (a.dim + 15) & ~15u, qp = DP + 8;
    const uint32_t g = lane >> 2, t2 = (lane & 3) * 2;
    const uint32_t base = s32(smem);
    float *pw = reinterpret_cast<float *>(smem + L.pw), *nst = reinterpret_cast<float *>(smem + L.nst), *raw = reinterpret_cast<float *>(smem + L.raw);
    auto bf = [&](uint32_t off) { return reinterpret_cast<__nv_bfloat16 *>(smem + off); };
    const uint32_t kb = a.H * a.dim, vb = 2 * kb, rs = 2 * a.dim + VCH;
    const bool with_n = GATED && blockIdx.x == 0, vec = a.dim % 4 == 0 && a.vdim % 4 == 0 && a.stride % 4 == 0;
    float *proj = a.proj + (size_t)s * a.R * a.stride;

    // a block's rows -> raw [64][q | k | v slice]
    auto stage = [&](uint32_t r0) {
        const uint32_t n = min(C, a.R - r0), nd = a.dim / 4;
        for (uint32_t r = warp; r < n; r += RT / 32) {
            const float *row = proj + (size_t)(r0 + r) * a.stride;
            const uint32_t dst = base + L.raw + r * rs * 4;
            for (uint32_t c = lane; c < 2 * nd + VCH / 4; c += 32) {
                const bool is_v = c >= 2 * nd;
                const uint32_t j = is_v ? (c - 2 * nd) * 4 : 0;
                const float *src = is_v ? row + vb + h * a.vdim + v0 + j : c < nd ? row + h * a.dim + c * 4 : row + kb + h * a.dim + (c - nd) * 4;
                const bool in = !is_v || j < nv;
                cp16(dst + c * 16, in ? src : row, in);
            }
        }
        cp_commit();
    };
    // the gates' projections of rows 2 lane, 2 lane + 1 of a block
    auto gate_rows = [&](uint32_t r0, float (&zi)[2], float (&zf)[2]) {
        const uint32_t n = min(C, a.R - r0);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const float *row = proj + (size_t)(r0 + min(2 * lane + e, n - 1)) * a.stride + 2 * a.H * (a.dim + a.vdim) + h;
            zi[e] = row[0];
            zf[e] = row[a.H];
        }
    };
    if (staged) stage(0);
    float zi[2], zf[2];
    if (GATED && warp == 0) gate_rows(0, zi, zf);

    // the state: registers, and its two parts in shared memory for Q S
    float st[ND][4][4];
    float *gst = state_of(a, s) + (size_t)h * a.dim * a.vdim + v0;
    auto state_parts = [&]() {
#pragma unroll
        for (int i = 0; i < ND; ++i) {
            const uint32_t d0 = (warp + 8 * i) * 16 + g;
            if ((warp + 8 * i) * 16 >= DP) continue;
#pragma unroll
            for (int n = 0; n < 4; ++n)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    uint32_t hi, lo;
                    split_pair(st[i][n][2 * e], st[i][n][2 * e + 1], hi, lo);
                    const uint32_t at = (d0 + 8 * e) * VP + n * 8 + t2;
                    *reinterpret_cast<uint32_t *>(bf(L.sh) + at) = hi;
                    *reinterpret_cast<uint32_t *>(bf(L.sl) + at) = lo;
                }
        }
    };
#pragma unroll
    for (int i = 0; i < ND; ++i)
#pragma unroll
        for (int n = 0; n < 4; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const uint32_t d = (warp + 8 * i) * 16 + g + (e >> 1) * 8, c = n * 8 + t2 + (e & 1);
                st[i][n][e] = d < a.dim && c < nv ? gst[(size_t)d * a.vdim + c] : 0.0f;
            }
    state_parts();
    float m0 = 0.0f;
    if constexpr (GATED) {
        m0 = state_m(a, s, h)[blockIdx.x];                       // this slice's own copy
        if (with_n)
            for (uint32_t d = tid; d < DP; d += RT) nst[d] = d < a.dim ? state_n(a, s, h)[d] : 0.0f;
    } else {
        for (uint32_t i = tid; i <= C; i += RT) pw[i] = a.powers[h * (C + 1) + i];
    }

    for (uint32_t r0 = 0; r0 < a.R; r0 += C) {
        const uint32_t n = min(C, a.R - r0);
        float *rows = proj + (size_t)r0 * a.stride;
        if (staged) cp_wait<0>();
        __syncthreads();                                         // the raw rows are here; the last block's operands are free
        if constexpr (GATED) {
            if (warp == 0) {
                block_gates(a, h, lane, m0, zi, zf, bg);
                if (r0 + C < a.R) gate_rows(r0 + C, zi, zf);
            }
        } else if (r0 == 0 && tid < C) {
            bg.rowf[tid] = pw[tid + 1];
        }
        auto load4 = [&](const float *p, uint32_t i, uint32_t lim) -> float4 {
            if (vec) return i < lim ? *reinterpret_cast<const float4 *>(p + i) : make_float4(0.f, 0.f, 0.f, 0.f);
            return make_float4(i < lim ? p[i] : 0.f, i + 1 < lim ? p[i + 1] : 0.f, i + 2 < lim ? p[i + 2] : 0.f, i + 3 < lim ? p[i + 3] : 0.f);
        };
        auto put4 = [&](uint32_t hi_off, uint32_t lo_off, uint32_t at, const float4 &v) {
            uint2 hi, lo;
            split_pair(v.x, v.y, hi.x, lo.x);
            split_pair(v.z, v.w, hi.y, lo.y);
            *reinterpret_cast<uint2 *>(bf(hi_off) + at) = hi;
            *reinterpret_cast<uint2 *>(bf(lo_off) + at) = lo;
        };
        auto act4 = [&](float4 v, float sc) {
            if (a.act) { v.x = silu(v.x); v.y = silu(v.y); v.z = silu(v.z); v.w = silu(v.w); }
            v.x *= sc; v.y *= sc; v.z *= sc; v.w *= sc;
            return v;
        };
#pragma unroll 2
        for (uint32_t r = warp; r < C; r += RT / 32)
            for (uint32_t d = lane * 4; d < DP; d += 128) {
                const float *q = staged ? raw + r * rs : rows + (size_t)r * a.stride + h * a.dim, *k = staged ? q + a.dim : q + kb;
                const float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
                const float4 q4 = r < n ? load4(q, d, a.dim) : z, k4 = r < n ? load4(k, d, a.dim) : z;
                put4(L.qh, L.ql, r * qp + d, act4(q4, a.qscale));
                put4(L.kh, L.kl, r * qp + d, act4(k4, a.kscale));
            }
        __syncthreads();                                         // Q, K and the gates are there
        {   // v, and v times its row's weight in the outgoing state: 8 columns per thread
            const uint32_t r = tid >> 2, c = (tid & 3) * 8;
            float w = 0.0f;
            if (r < n) w = GATED ? expf((float)(bg.rowd(n - 1) + bg.cold(r))) : pw[n - 1 - r];
            const float *v = staged ? raw + r * rs + 2 * a.dim : rows + (size_t)r * a.stride + vb + h * a.vdim + v0;
#pragma unroll
            for (int i = 0; i < 8; i += 4) {
                const float4 v4 = act4(r < n ? load4(v, c + i, nv) : make_float4(0.f, 0.f, 0.f, 0.f), 1.0f);
                put4(L.vh, L.vl, r * VP + c + i, v4);
                put4(L.wh, L.wl, r * VP + c + i, make_float4(v4.x * w, v4.y * w, v4.z * w, v4.w * w));
            }
        }
        const uint32_t mt = warp & 3, half = warp >> 2;          // row tile; which half of the columns
        const uint32_t a_row = (mt * 16 + (lane & 15)) * qp + (lane >> 4) * 8;
        if (half * 32 < mt * 16 + 16) {                          // scores [16 x 32] on or below the diagonal
            float acc[4][4] = {};
            for (uint32_t k = 0; k < DP; k += 16) {
                uint32_t ah[4], al[4];
                ldsm4(ah, base + L.qh + (a_row + k) * 2);
                ldsm4(al, base + L.ql + (a_row + k) * 2);
#pragma unroll
                for (int p = 0; p < 2; ++p) {
                    uint32_t bh[4], bl[4];
                    const uint32_t at = ((half * 32 + p * 16 + (lane & 7) + ((lane >> 4) << 3)) * qp + k + ((lane >> 3) & 1) * 8) * 2;
                    ldsm4(bh, base + L.kh + at);
                    ldsm4(bl, base + L.kl + at);
                    mma3(acc[2 * p], ah, al, bh, bl);
                    mma3(acc[2 * p + 1], ah, al, bh + 2, bl + 2);
                }
            }
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const uint32_t ri = mt * 16 + g + 8 * e;
                const double rd = GATED ? bg.rowd(ri) : 0.0;
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const uint32_t cj = half * 32 + j * 8 + t2;
                    float p[2];
#pragma unroll
                    for (int i = 0; i < 2; ++i)
                        p[i] = cj + i <= ri ? acc[j][2 * e + i] * (GATED ? expf((float)(rd + bg.cold(cj + i))) : pw[ri - cj - i]) : 0.0f;
                    uint32_t hi, lo;
                    split_pair(p[0], p[1], hi, lo);
                    *reinterpret_cast<uint32_t *>(bf(L.ph) + ri * PP + cj) = hi;
                    *reinterpret_cast<uint32_t *>(bf(L.pl) + ri * PP + cj) = lo;
                }
            }
        }
        float o[2][4] = {};                                      // output [16 x 16]: row tile mt, columns 16 half ..
        const uint32_t b_col = half * 16 + (lane >> 4) * 8;
        for (uint32_t k = 0; k < DP; k += 16) {
            uint32_t ah[4], al[4], bh[4], bl[4];
            ldsm4(ah, base + L.qh + (a_row + k) * 2);
            ldsm4(al, base + L.ql + (a_row + k) * 2);
            const uint32_t at = ((k + (lane & 15)) * VP + b_col) * 2;
            ldsm4t(bh, base + L.sh + at);
            ldsm4t(bl, base + L.sl + at);
            mma3(o[0], ah, al, bh, bl);
            mma3(o[1], ah, al, bh + 2, bl + 2);
        }
        {
            const float f0 = bg.rowf[mt * 16 + g], f1 = bg.rowf[mt * 16 + g + 8];
#pragma unroll
            for (int j = 0; j < 2; ++j) { o[j][0] *= f0; o[j][1] *= f0; o[j][2] *= f1; o[j][3] *= f1; }
        }
        __syncthreads();                                         // P, V, wV are there; the raw rows and S are free
        if (staged && r0 + C < a.R) stage(r0 + C);
        for (uint32_t k = 0; k <= mt; ++k) {                     // P is zero right of the diagonal tile
            uint32_t ah[4], al[4], bh[4], bl[4];
            const uint32_t pa = ((mt * 16 + (lane & 15)) * PP + k * 16 + (lane >> 4) * 8) * 2, at = ((k * 16 + (lane & 15)) * VP + b_col) * 2;
            ldsm4(ah, base + L.ph + pa);
            ldsm4(al, base + L.pl + pa);
            ldsm4t(bh, base + L.vh + at);
            ldsm4t(bl, base + L.vl + at);
            mma3(o[0], ah, al, bh, bl);
            mma3(o[1], ah, al, bh + 2, bl + 2);
        }
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const uint32_t r = mt * 16 + g + 8 * e, c = half * 16 + j * 8 + t2;
                float *dst = rows + (size_t)r * a.stride + vb + h * a.vdim + v0 + c;
                if (r >= n) continue;
                if (vec && c < nv) *reinterpret_cast<float2 *>(dst) = make_float2(o[j][2 * e], o[j][2 * e + 1]);
                else {
                    if (c < nv) dst[0] = o[j][2 * e];
                    if (c + 1 < nv) dst[1] = o[j][2 * e + 1];
                }
            }
        const float keep = GATED ? bg.rowf[n - 1] : pw[n];
#pragma unroll
        for (int i = 0; i < ND; ++i) {
            const uint32_t d0 = (warp + 8 * i) * 16;
            if (d0 >= DP) continue;
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) st[i][j][e] *= keep;
            for (uint32_t k = 0; k < C; k += 16) {
                uint32_t ah[4], al[4];
                const uint32_t ka = ((k + (lane & 7) + ((lane >> 4) << 3)) * qp + d0 + ((lane >> 3) & 1) * 8) * 2;
                ldsm4t(ah, base + L.kh + ka);
                ldsm4t(al, base + L.kl + ka);
#pragma unroll
                for (int p = 0; p < 2; ++p) {
                    uint32_t bh[4], bl[4];
                    const uint32_t at = ((k + (lane & 15)) * VP + p * 16 + (lane >> 4) * 8) * 2;
                    ldsm4t(bh, base + L.wh + at);
                    ldsm4t(bl, base + L.wl + at);
                    mma3(st[i][2 * p], ah, al, bh, bl);
                    mma3(st[i][2 * p + 1], ah, al, bh + 2, bl + 2);
                }
            }
        }
        state_parts();
        if constexpr (GATED) {
            const float m_end = bg.m[n - 1];
            if (with_n) {
                {   // n . q: four threads per row
                    const uint32_t r = tid >> 2, p = tid & 3;
                    float nq = 0.0f, ps = 0.0f;
                    for (uint32_t d = p * 2; d < DP; d += 8) {
                        const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(bf(L.qh) + r * qp + d));
                        const float2 y = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(bf(L.ql) + r * qp + d));
                        nq = fmaf(x.x + y.x, nst[d], fmaf(x.y + y.y, nst[d + 1], nq));
                    }
                    for (uint32_t j = p * 2; j < (r / 16 + 1) * 16; j += 8) {
                        const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(bf(L.ph) + r * PP + j));
                        const float2 y = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(bf(L.pl) + r * PP + j));
                        ps += (x.x + y.x) + (x.y + y.y);
                    }
                    nq = fmaf(nq, bg.rowf[r], ps);
                    nq += __shfl_xor_sync(0xffffffffu, nq, 1);
                    nq += __shfl_xor_sync(0xffffffffu, nq, 2);
                    if (p == 0 && r < n) {
                        float *aux = a.row_aux + (((size_t)s * a.R + r0 + r) * a.H + h) * 2;
                        aux[0] = nq;
                        aux[1] = bg.m[r];
                    }
                }
                if (tid < C) pw[tid] = tid < n ? expf((float)(bg.rowd(n - 1) + bg.cold(tid))) : 0.0f;
                __syncthreads();
                for (uint32_t d = tid; d < DP; d += RT) {
                    float v = nst[d] * keep;
#pragma unroll 4
                    for (uint32_t j = 0; j < n; ++j)
                        v = fmaf(pw[j], __bfloat162float(bf(L.kh)[j * qp + d]) + __bfloat162float(bf(L.kl)[j * qp + d]), v);
                    nst[d] = v;
                }
            }
            m0 = m_end;
        }
    }
#pragma unroll
    for (int i = 0; i < ND; ++i)
#pragma unroll
        for (int n = 0; n < 4; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const uint32_t d = (warp + 8 * i) * 16 + g + (e >> 1) * 8, c = n * 8 + t2 + (e & 1);
                if (d < a.dim && c < nv) gst[(size_t)d * a.vdim + c] = st[i][n][e];
            }
    if constexpr (GATED) {
        if (tid == 0) state_m(a, s, h)[blockIdx.x] = m0;
        if (with_n)
            for (uint32_t d = tid; d < a.dim; d += RT) state_n(a, s, h)[d] = nst[d];       // (a thread's own elements)
    }
}

constexpr uint32_t SMEM_LIMIT = 225 * 1024;

template <bool GATED, int ND>
int launch(qb_ctx *ctx, const QbRecurrence &a) {
    const bool vec = a.dim % 4 == 0 && a.vdim % 4 == 0 && a.stride % 4 == 0;
    const uint32_t staged = vec && mma_smem(a.dim, 1).total <= SMEM_LIMIT, smem = mma_smem(a.dim, staged).total;
    QB_CUDA(cudaFuncSetAttribute(recurrence_mma_kernel<GATED, ND>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    QB_CUDA(qb_launch_pdl(ctx->stream, recurrence_mma_kernel<GATED, ND>, dim3(qb_recurrence_slices(a.vdim), a.H, a.ns), dim3(RT), (size_t)smem, a, staged));
    QB_LAUNCHED(ctx, GATED ? "gated_recurrence_mma_kernel" : "recurrence_mma_kernel");
    return QB_OK;
}

}  // namespace

bool qb_recurrence_mma_supports(const QbRecurrence &a) { return !a.out.f32 && a.dim <= 256 && mma_smem(a.dim, 0).total <= SMEM_LIMIT; }

int qb_launch_recurrence_mma(qb_ctx *ctx, const QbRecurrence &a) {
    if (a.gated) return a.dim <= 128 ? launch<true, 1>(ctx, a) : launch<true, 2>(ctx, a);
    return a.dim <= 128 ? launch<false, 1>(ctx, a) : launch<false, 2>(ctx, a);
}
