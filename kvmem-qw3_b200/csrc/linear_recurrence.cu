// Linear recurrences: a matrix state per head that decays and takes one outer product per token, read by a query, with a
// normalised and gated output; 32-bit state.
//   retention   S_t = decay S_(t-1) + k_t v_t^T, fixed decay per head, rotated q and k, rms per head, silu gate
//   lightning   the same with silu on q, k and v, no rotation, one rms over all heads with a weight, sigmoid gate
//   mLSTM       decay and input weight from exponential gates that each token computes, stabilised by a running maximum m, a
//               normaliser n beside the state: o = S^T q / (max(|n . q|, exp(-m)) + 1e-6)
// The constants and switches are fields of QbRecurrence.  GATED kernels are the form with gates of the token's own.
//
// Decode rows (recurrence_step_kernel, recurrence_decode_kernel): one launch takes the projections (adding their K-segment
// partial sums), activates or rotates q and k, advances the state and writes the gated output.  A CTA owns a slice of a
// head's value columns; the slices of a head form a thread-block cluster that adds up the head's mean square through
// distributed shared memory.
//
// Prompt chunks (recurrence_chunk_kernel): blocks of 64 rows.  With D[i][j] the decay from row j to row i,
//     O = (Q K^T . D) V + diag(a_i) Q S        S' = keep S + sum_j w_j k_j v_j^T
// everything in fp32 on the CUDA cores (float32 models), or on the tensor cores with operands split into two bfloat16 parts
// (linear_recurrence_mma.cu).  Fixed decays: powers from a table made in double precision.  Gated: with b the
// running sum of the log forget gates (double precision), m_i = max(m_0 + b_i, max_j (i_j + b_i - b_j)),
//     D[i][j] = exp(b_i - b_j + i_j - m_i)   a_i = exp(m_0 + b_i - m_i)   w_j = exp(b_n - b_j + i_j - m_n)   keep = a_n
// and the division by the normaliser waits for the output kernel.
#include "linear_recurrence.cuh"

#include <cooperative_groups.h>
namespace cg = cooperative_groups;

namespace {
using namespace qbrec;

constexpr int RT = 256;

// "This CTA runs": arrived at on entry, awaited before the first store into another CTA's shared memory, which must not be
// touched before that CTA has started.
__device__ __forceinline__ void cluster_started() { asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait_started() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }

template <typename T, bool GATED>
__global__ void __launch_bounds__(RT)
recurrence_step_kernel(QbRecurrence a, uint32_t vc) {
    cluster_started();
    QB_PDL_ENTER();
    cg::cluster_group cl = cg::this_cluster();
    extern __shared__ float sm[];
    float *st = sm;                               // [dim][vc]
    float *qs = st + (size_t)a.dim * vc, *ks = qs + a.dim;
    float *cs = ks + a.dim, *sn = cs + a.rot.dims / 2;
    float *red = sn + a.rot.dims / 2;             // [8][vc]
    float *nv_ = red + (RT / 32) * vc;            // gated: the normaliser [dim]
    __shared__ float xch[2][16], wsum[RT / 32];
    const uint32_t tid = threadIdx.x, h = blockIdx.y, s = blockIdx.z, v0 = blockIdx.x * vc;
    const uint32_t nv = min(vc, a.vdim - v0), rank = cl.block_rank(), csize = cl.num_blocks();
    const uint32_t rows = a.ns * a.R;
    const size_t ps = (size_t)rows * a.stride;
    float decay = GATED ? 1.0f : a.powers[h * (C + 1) + 1], add = 1.0f, m_run = 0.0f;
    float *gst = state_of(a, s) + (size_t)h * a.dim * a.vdim + v0;
    if constexpr (GATED) {
        m_run = state_m(a, s, h)[0];
        for (uint32_t d = tid; d < a.dim; d += RT) nv_[d] = state_n(a, s, h)[d];
    }
    for (uint32_t i = tid; i < a.dim * vc; i += RT) {
        const uint32_t d = i / vc, c = i % vc;
        st[i] = c < nv ? gst[(size_t)d * a.vdim + c] : 0.0f;
    }
    const uint32_t kb = a.H * a.dim, vb = 2 * kb, gb = vb + a.H * a.vdim;
    const uint32_t half = a.rot.dims / 2;
    for (uint32_t r = 0; r < a.R; ++r) {
        const size_t m = (size_t)s * a.R + r, base = m * a.stride;
        const int pos = a.seq_pos[s] + (int)r;
        for (uint32_t i = tid; i < half; i += RT) qb_rot_angle(a.rot, pos, i, cs[i], sn[i]);
        __syncthreads();
        for (uint32_t d = tid; d < a.dim; d += RT) {
            float q = qb_sum8(a.proj, base + h * a.dim + d, a.S, ps), k = qb_sum8(a.proj, base + kb + h * a.dim + d, a.S, ps);
            if (d < a.rot.dims) {
                uint32_t i, p; bool first;
                qb_rot_pair(a.rot, d, i, p, first);
                const float q2 = qb_sum8(a.proj, base + h * a.dim + p, a.S, ps), k2 = qb_sum8(a.proj, base + kb + h * a.dim + p, a.S, ps);
                q = first ? q * cs[i] - q2 * sn[i] : q * cs[i] + q2 * sn[i];
                k = first ? k * cs[i] - k2 * sn[i] : k * cs[i] + k2 * sn[i];
            }
            qs[d] = act_in(a, q) * a.qscale;
            ks[d] = act_in(a, k) * a.kscale;
        }
        float nq = 0.0f;
        if constexpr (GATED) {                       // every thread works out the same gates
            const StepGates g = step_gates(a, h, base, ps, m_run);
            decay = g.keep; add = g.add; m_run = g.m;
            for (uint32_t d = tid; d < a.dim; d += RT) {      // (a thread reads back its own qs, ks)
                ks[d] *= add;
                nv_[d] = fmaf(nv_[d], decay, ks[d]);
                nq = fmaf(nv_[d], qs[d], nq);
            }
            nq = qb_block_sum(nq, wsum, RT / 32);
        }
        __syncthreads();
        const uint32_t rg = tid >> 5;
        for (uint32_t c = tid & 31; c < vc; c += 32) {
            const float v = c < nv ? act_in(a, qb_sum8(a.proj, base + vb + h * a.vdim + v0 + c, a.S, ps)) : 0.0f;
            float o = 0.0f;
#pragma unroll 4
            for (uint32_t d = rg; d < a.dim; d += RT / 32) {
                const float t = fmaf(st[d * vc + c], decay, ks[d] * v);
                st[d * vc + c] = t;
                o = fmaf(t, qs[d], o);
            }
            red[rg * vc + c] = o;
        }
        __syncthreads();
        if (r == 0) cluster_wait_started();
        if (tid < 32) {
            float ss = 0.0f;
            for (uint32_t c = tid; c < vc; c += 32) {
                float o = 0.0f;
#pragma unroll
                for (uint32_t g = 0; g < RT / 32; ++g) o += red[g * vc + c];
                if constexpr (GATED) o /= normaliser(nq, m_run);
                red[c] = o;
                ss += o * o;
            }
            ss = warp_sum(ss);
            if (tid < csize) cl.map_shared_rank(&xch[0][0], tid)[(r & 1) * 16 + rank] = ss;
        }
        cl.sync();                                   // every slice's sum is here (and red[] within the CTA)
        float tot = 0.0f;
        for (uint32_t i = 0; i < csize; ++i) tot += xch[r & 1][i];
        if (a.row_ss && rank == 0 && tid == 0) a.row_ss[m * a.H + h] = tot;
        const float inv = a.row_ss ? 1.0f : rsqrtf(tot / (float)a.vdim + a.eps);
        T *out = (T *)a.out.p + m * a.out.ld + h * a.vdim + v0;
        for (uint32_t c = tid; c < nv; c += RT) {
            const float g = qb_sum8(a.proj, base + gb + h * a.vdim + v0 + c, a.S, ps);
            out[c] = qb_cast<T>(red[c] * inv * (a.norm_w ? a.norm_w[h * a.vdim + v0 + c] : 1.0f) * gate_out(a, g));
        }
        __syncthreads();
    }
    for (uint32_t i = tid; i < a.dim * vc; i += RT) {
        const uint32_t d = i / vc, c = i % vc;
        if (c < nv) gst[(size_t)d * a.vdim + c] = st[i];
    }
    if constexpr (GATED)                             // (every slice read n and m before the first row's cluster barrier)
        if (rank == 0) {
            for (uint32_t d = tid; d < a.dim; d += RT) state_n(a, s, h)[d] = nv_[d];
            if (tid < qb_recurrence_slices(a.vdim)) state_m(a, s, h)[tid] = m_run;
        }
    cl.sync();                                       // no CTA leaves while a peer may still write its xch
}

// One row per sequence (plain decode): the state never leaves the registers -- a thread holds NI pieces of four value
// columns, all requested at once before the row's q and k are rotated.  Needs vdim and the projection offsets to be
// multiples of 4.
template <typename T, int NI, bool GATED>
__global__ void __launch_bounds__(RT)
recurrence_decode_kernel(QbRecurrence a, uint32_t vc) {
    cluster_started();
    QB_PDL_ENTER();
    cg::cluster_group cl = cg::this_cluster();
    extern __shared__ float sm[];
    float *qs = sm, *ks = qs + a.dim;
    float4 *red = reinterpret_cast<float4 *>(ks + a.dim);      // [RT / 32 warps][vc / 4]   (dim is even: 16-byte aligned)
    __shared__ float xch[16], part[RT / 32], npart[RT / 32];
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y, m = blockIdx.z, v0 = blockIdx.x * vc;
    const uint32_t nv = min(vc, a.vdim - v0), g4 = vc / 4, c4 = tid % g4, dg = tid / g4, nd = RT / g4;
    const size_t base = (size_t)m * a.stride, ps = (size_t)a.ns * a.stride;
    const bool on = c4 * 4 < nv;
    float *gst = state_of(a, m) + (size_t)h * a.dim * a.vdim + v0 + c4 * 4;
    float4 st[NI];
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const uint32_t d = dg + i * nd;
        st[i] = on && d < a.dim ? *reinterpret_cast<const float4 *>(gst + (size_t)d * a.vdim) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const uint32_t kb = a.H * a.dim, vb = 2 * kb, gb = vb + a.H * a.vdim;
    StepGates g{1.0f, 1.0f, 0.0f};
    if constexpr (GATED) g = step_gates(a, h, base, ps, state_m(a, m, h)[0]);
    const float decay = GATED ? g.keep : a.powers[h * (C + 1) + 1];
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (on) {
        const float *p = a.proj + base + vb + h * a.vdim + v0 + c4 * 4;
        v = *reinterpret_cast<const float4 *>(p);
        for (uint32_t s = 1; s < a.S; ++s) {
            const float4 w = *reinterpret_cast<const float4 *>(p + s * ps);
            v.x += w.x; v.y += w.y; v.z += w.z; v.w += w.w;
        }
        v.x = act_in(a, v.x); v.y = act_in(a, v.y); v.z = act_in(a, v.z); v.w = act_in(a, v.w);
    }
    const int pos = a.seq_pos[m];
    for (uint32_t t = tid; t < 2 * a.dim; t += RT) {           // q, then k: a pair's two threads each take one element
        const bool is_k = t >= a.dim;
        const uint32_t d = is_k ? t - a.dim : t;
        const size_t at = base + (is_k ? kb : 0) + h * a.dim;
        float u = qb_sum8(a.proj, at + d, a.S, ps);
        if (d < a.rot.dims) {
            uint32_t i, p; bool first;
            qb_rot_pair(a.rot, d, i, p, first);
            const float w = qb_sum8(a.proj, at + p, a.S, ps);
            float c, sn;
            qb_rot_angle(a.rot, pos, i, c, sn);
            u = first ? u * c - w * sn : u * c + w * sn;
        }
        u = act_in(a, u);
        sm[t] = is_k ? u * a.kscale * g.add : u * a.qscale;
    }
    __syncthreads();
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const uint32_t d = dg + i * nd;
        if (d < a.dim) {
            const float q = qs[d], k = ks[d];
            st[i].x = fmaf(st[i].x, decay, k * v.x); st[i].y = fmaf(st[i].y, decay, k * v.y);
            st[i].z = fmaf(st[i].z, decay, k * v.z); st[i].w = fmaf(st[i].w, decay, k * v.w);
            if (on) *reinterpret_cast<float4 *>(gst + (size_t)d * a.vdim) = st[i];
            o.x = fmaf(st[i].x, q, o.x); o.y = fmaf(st[i].y, q, o.y); o.z = fmaf(st[i].z, q, o.z); o.w = fmaf(st[i].w, q, o.w);
        }
    }
    for (uint32_t off = g4; off < 32; off <<= 1) {             // lanes of a warp that hold the same columns
        o.x += __shfl_xor_sync(0xffffffffu, o.x, off); o.y += __shfl_xor_sync(0xffffffffu, o.y, off);
        o.z += __shfl_xor_sync(0xffffffffu, o.z, off); o.w += __shfl_xor_sync(0xffffffffu, o.w, off);
    }
    if (lane < g4) red[warp * g4 + lane] = o;
    if constexpr (GATED) {
        const float *n = state_n(a, m, h);
        float nq = 0.0f;
        for (uint32_t d = tid; d < a.dim; d += RT) nq = fmaf(fmaf(n[d], decay, ks[d]), qs[d], nq);
        nq = warp_sum(nq);
        if (lane == 0) npart[warp] = nq;
    }
    __syncthreads();
    float out = 0.0f;
    if (tid < vc) {
        const float *r = reinterpret_cast<const float *>(red);
#pragma unroll
        for (uint32_t w = 0; w < RT / 32; ++w) out += r[w * vc + tid];
    }
    if constexpr (GATED) {
        float nq = 0.0f;
#pragma unroll
        for (uint32_t w = 0; w < RT / 32; ++w) nq += npart[w];
        out /= normaliser(nq, g.m);
    }
    const float ss = warp_sum(out * out);                       // columns past vdim are zero
    if (lane == 0) part[warp] = ss;
    __syncthreads();
    const uint32_t csize = cl.num_blocks();
    float tot = 0.0f;
#pragma unroll
    for (uint32_t w = 0; w < RT / 32; ++w) tot += part[w];
    cluster_wait_started();
    if (csize > 1) {
        if (tid < csize) cl.map_shared_rank(xch, tid)[cl.block_rank()] = tot;
        cl.sync();
        tot = 0.0f;
        for (uint32_t i = 0; i < csize; ++i) tot += xch[i];
    }
    if constexpr (GATED)                                         // every slice has read n and m (the cluster barrier, or no other slice)
        if (cl.block_rank() == 0) {
            float *n = state_n(a, m, h);
            for (uint32_t d = tid; d < a.dim; d += RT) n[d] = fmaf(n[d], decay, ks[d]);
            if (tid < qb_recurrence_slices(a.vdim)) state_m(a, m, h)[tid] = g.m;
        }
    if (a.row_ss && cl.block_rank() == 0 && tid == 0) a.row_ss[(size_t)m * a.H + h] = tot;
    const float inv = a.row_ss ? 1.0f : rsqrtf(tot / (float)a.vdim + a.eps);
    if (tid < nv) {
        const uint32_t c = h * a.vdim + v0 + tid;
        const float z = qb_sum8(a.proj, base + gb + c, a.S, ps);
        ((T *)a.out.p + (size_t)m * a.out.ld)[c] = qb_cast<T>(out * inv * (a.norm_w ? a.norm_w[c] : 1.0f) * gate_out(a, z));
    }
}

// A prompt chunk's projections in place: K-segment partial sums added, q and k rotated.
__global__ void __launch_bounds__(RT)
recurrence_rotate_kernel(QbRecurrence a) {
    QB_PDL_ENTER();
    extern __shared__ float sm[];
    const uint32_t m = blockIdx.x, half = a.rot.dims / 2, s = m / a.R;
    float *cs = sm, *sn = sm + half;
    const int pos = a.seq_pos[s] + (int)(m % a.R);
    for (uint32_t i = threadIdx.x; i < half; i += RT) qb_rot_angle(a.rot, pos, i, cs[i], sn[i]);
    __syncthreads();
    const size_t base = (size_t)m * a.stride, ps = (size_t)a.ns * a.R * a.stride;
    float *row = a.proj + base;
    // rotated pairs
    for (uint32_t t = threadIdx.x; t < 2 * a.H * half; t += RT) {
        const uint32_t i = t % half, hh = t / half;                           // hh < H: q heads, then k heads
        const uint32_t j = hh * a.dim + (a.rot.interleaved ? 2 * i : i), p = a.rot.interleaved ? j + 1 : j + half;
        const float u = qb_sum8(a.proj, base + j, a.S, ps), v = qb_sum8(a.proj, base + p, a.S, ps);
        row[j] = u * cs[i] - v * sn[i];
        row[p] = v * cs[i] + u * sn[i];
    }
    if (a.S == 1) return;
    // dimensions that pass, and the columns behind q and k
    const uint32_t rest = a.dim - a.rot.dims;
    for (uint32_t t = threadIdx.x; t < 2 * a.H * rest; t += RT) {
        const uint32_t hh = t / rest, j = hh * a.dim + a.rot.dims + t % rest;
        row[j] = qb_sum8(a.proj, base + j, a.S, ps);
    }
    for (uint32_t j = 2 * a.H * a.dim + threadIdx.x; j < a.stride; j += RT) row[j] = qb_sum8(a.proj, base + j, a.S, ps);
}

// grid (value slices, H, sequences).  q and k are rotated; the outputs replace the v columns of the projection.  Gated: the
// first slice also advances n and leaves n . q and m of every row in row_aux.
template <bool GATED>
__global__ void __launch_bounds__(RT)
recurrence_chunk_kernel(QbRecurrence a, uint32_t dimr) {
    QB_PDL_ENTER();
    extern __shared__ float4 sm4[];
    float *sm = reinterpret_cast<float *>(sm4);
    const uint32_t dp = dimr + 4;
    constexpr uint32_t PP = C + 4;
    float *qs = sm, *ks = qs + C * dp, *vs = ks + C * dp, *st = vs + C * VCH, *pm = st + dimr * VCH, *pw = pm + C * PP;
    float *nst = pw + C + 4;                      // gated: n [dimr]
    // per block: factor of the incoming state per row (bg.rowf), weight of a row in the outgoing state
    __shared__ BlockGates bg;
    __shared__ float colf[C], keep_s;
    const uint32_t tid = threadIdx.x, h = blockIdx.y, s = blockIdx.z, v0 = blockIdx.x * VCH;
    const uint32_t nv = min(VCH, a.vdim - v0);
    float *gst = state_of(a, s) + (size_t)h * a.dim * a.vdim + v0;
    for (uint32_t i = tid; i < dimr * VCH; i += RT) {
        const uint32_t d = i / VCH, c = i % VCH;
        st[i] = (d < a.dim && c < nv) ? gst[(size_t)d * a.vdim + c] : 0.0f;
    }
    const bool with_n = GATED && blockIdx.x == 0;
    float m0 = 0.0f;
    if constexpr (GATED) {
        m0 = state_m(a, s, h)[blockIdx.x];                       // this slice's own copy
        if (with_n)
            for (uint32_t d = tid; d < dimr; d += RT) nst[d] = d < a.dim ? state_n(a, s, h)[d] : 0.0f;
    } else {
        for (uint32_t i = tid; i <= C; i += RT) pw[i] = a.powers[h * (C + 1) + i];
        __syncthreads();
    }
    const uint32_t kb = a.H * a.dim, vb = 2 * kb;
    for (uint32_t r0 = 0; r0 < a.R; r0 += C) {
        const uint32_t n = min(C, a.R - r0);
        float *rows = a.proj + ((size_t)s * a.R + r0) * a.stride;
        for (uint32_t i = tid; i < C * dimr; i += RT) {
            const uint32_t r = i / dimr, d = i % dimr;
            const bool in = r < n && d < a.dim;
            qs[r * dp + d] = in ? rows[(size_t)r * a.stride + h * a.dim + d] : 0.0f;
            ks[r * dp + d] = in ? rows[(size_t)r * a.stride + kb + h * a.dim + d] : 0.0f;
        }
        for (uint32_t i = tid; i < C * VCH; i += RT) {
            const uint32_t r = i / VCH, c = i % VCH;
            vs[i] = (r < n && c < nv) ? rows[(size_t)r * a.stride + vb + h * a.vdim + v0 + c] : 0.0f;
        }
        if (a.act || a.qscale != 1.0f || a.kscale != 1.0f) {     // (a thread's own elements; silu(0) = 0)
            for (uint32_t i = tid; i < C * dimr; i += RT) {
                const uint32_t at = i / dimr * dp + i % dimr;
                qs[at] = act_in(a, qs[at]) * a.qscale;
                ks[at] = act_in(a, ks[at]) * a.kscale;
            }
            if (a.act) for (uint32_t i = tid; i < C * VCH; i += RT) vs[i] = act_in(a, vs[i]);
        }
        if constexpr (GATED) {
            if (tid < 32) {
                const uint32_t gi = 2 * a.H * (a.dim + a.vdim) + h;
                float zi[2], zf[2];
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const float *row = rows + (size_t)min(2 * tid + e, n - 1) * a.stride + gi;
                    zi[e] = row[0];
                    zf[e] = row[a.H];
                }
                block_gates(a, h, tid, m0, zi, zf, bg);
            }
            __syncthreads();
            if (tid < C) {
                colf[tid] = tid < n ? expf((float)(bg.rowd(n - 1) + bg.cold(tid))) : 0.0f;
                if (tid == 0) keep_s = bg.rowf[n - 1];
            }
            m0 = bg.m[n - 1];
        } else if (tid < C) {
            bg.rowf[tid] = pw[tid + 1];
            colf[tid] = tid < n ? pw[n - 1 - tid] : 0.0f;
            if (tid == 0) keep_s = pw[n];
        }
        __syncthreads();
        {   // decayed scores
            const uint32_t tx = tid & 15, ty = tid >> 4;
            float acc[4][4] = {};
            for (uint32_t d = 0; d < dimr; d += 4) {
                float4 q[4], k[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    q[i] = *reinterpret_cast<const float4 *>(qs + (ty * 4 + i) * dp + d);
                    k[i] = *reinterpret_cast<const float4 *>(ks + (tx + 16 * i) * dp + d);
                }
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int j = 0; j < 4; ++j)
                        acc[i][j] = fmaf(q[i].x, k[j].x, fmaf(q[i].y, k[j].y, fmaf(q[i].z, k[j].z, fmaf(q[i].w, k[j].w, acc[i][j]))));
            }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const uint32_t ri = ty * 4 + i, cj = tx + 16 * j;
                    if constexpr (GATED)
                        pm[ri * PP + cj] = cj <= ri ? acc[i][j] * expf((float)(bg.rowd(ri) + bg.cold(cj))) : 0.0f;
                    else
                        pm[ri * PP + cj] = cj <= ri ? acc[i][j] * pw[ri - cj] : 0.0f;
                }
        }
        __syncthreads();
        {   // outputs: rows r, r + 32; four columns
            const uint32_t c = (tid & 7) * 4, r = tid >> 3;
            float o[2][4] = {};
            for (uint32_t d = 0; d < dimr; d += 4) {
                float4 sv[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) sv[i] = *reinterpret_cast<const float4 *>(st + (d + i) * VCH + c);
#pragma unroll
                for (int k = 0; k < 2; ++k) {
                    const float4 q = *reinterpret_cast<const float4 *>(qs + (r + 32 * k) * dp + d);
                    const float qa[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        o[k][0] = fmaf(qa[i], sv[i].x, o[k][0]); o[k][1] = fmaf(qa[i], sv[i].y, o[k][1]);
                        o[k][2] = fmaf(qa[i], sv[i].z, o[k][2]); o[k][3] = fmaf(qa[i], sv[i].w, o[k][3]);
                    }
                }
            }
#pragma unroll
            for (int k = 0; k < 2; ++k)
#pragma unroll
                for (int i = 0; i < 4; ++i) o[k][i] *= bg.rowf[r + 32 * k];
            for (uint32_t j = 0; j < C; j += 4) {
                float4 vv[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) vv[i] = *reinterpret_cast<const float4 *>(vs + (j + i) * VCH + c);
#pragma unroll
                for (int k = 0; k < 2; ++k) {
                    const float4 p = *reinterpret_cast<const float4 *>(pm + (r + 32 * k) * PP + j);
                    const float pa[4] = {p.x, p.y, p.z, p.w};
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        o[k][0] = fmaf(pa[i], vv[i].x, o[k][0]); o[k][1] = fmaf(pa[i], vv[i].y, o[k][1]);
                        o[k][2] = fmaf(pa[i], vv[i].z, o[k][2]); o[k][3] = fmaf(pa[i], vv[i].w, o[k][3]);
                    }
                }
            }
#pragma unroll
            for (int k = 0; k < 2; ++k)
#pragma unroll
                for (int i = 0; i < 4; ++i)
                    if (r + 32 * k < n && c + i < nv) rows[(size_t)(r + 32 * k) * a.stride + vb + h * a.vdim + v0 + c + i] = o[k][i];
        }
        if (with_n) {                                            // n . q: four threads per row
            const uint32_t r = tid >> 2, p = tid & 3;
            float nq = 0.0f, ps = 0.0f;
            for (uint32_t d = p; d < dimr; d += 4) nq = fmaf(qs[r * dp + d], nst[d], nq);
            for (uint32_t j = p; j < C; j += 4) ps += pm[r * PP + j];
            nq = fmaf(nq, bg.rowf[r], ps);
            nq += __shfl_xor_sync(0xffffffffu, nq, 1);
            nq += __shfl_xor_sync(0xffffffffu, nq, 2);
            if (p == 0 && r < n) {
                float *aux = a.row_aux + (((size_t)s * a.R + r0 + r) * a.H + h) * 2;
                aux[0] = nq;
                aux[1] = bg.m[r];
            }
        }
        __syncthreads();
        if (with_n)
            for (uint32_t d = tid; d < dimr; d += RT) {
                float v = nst[d] * keep_s;
                for (uint32_t j = 0; j < n; ++j) v = fmaf(colf[j], ks[j * dp + d], v);
                nst[d] = v;
            }
        for (uint32_t t = tid; t < dimr * 2; t += RT) {      // state: four key dims x four columns
            const uint32_t d = (t >> 3) * 4, c = (t & 7) * 4;
            float acc[4][4];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int k = 0; k < 4; ++k) acc[i][k] = st[(d + i) * VCH + c + k] * keep_s;
            for (uint32_t j = 0; j < n; ++j) {
                const float w = colf[j];
                float4 v = *reinterpret_cast<const float4 *>(vs + j * VCH + c);
                const float4 k = *reinterpret_cast<const float4 *>(ks + j * dp + d);
                v.x *= w; v.y *= w; v.z *= w; v.w *= w;
                const float ka[4] = {k.x, k.y, k.z, k.w};
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    acc[i][0] = fmaf(ka[i], v.x, acc[i][0]); acc[i][1] = fmaf(ka[i], v.y, acc[i][1]);
                    acc[i][2] = fmaf(ka[i], v.z, acc[i][2]); acc[i][3] = fmaf(ka[i], v.w, acc[i][3]);
                }
            }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int k = 0; k < 4; ++k) st[(d + i) * VCH + c + k] = acc[i][k];
        }
        __syncthreads();
    }
    for (uint32_t i = tid; i < a.dim * VCH; i += RT) {
        const uint32_t d = i / VCH, c = i % VCH;
        if (c < nv) gst[(size_t)d * a.vdim + c] = st[i];
    }
    if constexpr (GATED) {
        if (tid == 0) state_m(a, s, h)[blockIdx.x] = m0;
        if (with_n)
            for (uint32_t d = tid; d < a.dim; d += RT) state_n(a, s, h)[d] = nst[d];
    }
}

// One warp per (row, head): normaliser, root mean square (or its sum of squares, where one norm spans the heads), weight, gate.
template <typename T, bool GATED>
__global__ void __launch_bounds__(RT)
recurrence_gate_kernel(QbRecurrence a) {
    QB_PDL_ENTER();
    const uint32_t t = blockIdx.x * (RT / 32) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (t >= a.ns * a.R * a.H) return;
    const uint32_t m = t / a.H, h = t % a.H;
    const float *o = a.proj + (size_t)m * a.stride + 2 * a.H * a.dim + h * a.vdim, *g = o + a.H * a.vdim;
    float den = 1.0f, ss = 0.0f;
    if constexpr (GATED) den = normaliser(a.row_aux[(size_t)t * 2], a.row_aux[(size_t)t * 2 + 1]);
    for (uint32_t c = lane; c < a.vdim; c += 32) { const float v = GATED ? o[c] / den : o[c]; ss += v * v; }
    ss = warp_sum(ss);
    if (a.row_ss && lane == 0) a.row_ss[t] = ss;
    const float inv = a.row_ss ? 1.0f : rsqrtf(ss / (float)a.vdim + a.eps);
    T *out = (T *)a.out.p + (size_t)m * a.out.ld + h * a.vdim;
    for (uint32_t c = lane; c < a.vdim; c += 32)
        out[c] = qb_cast<T>((GATED ? o[c] / den : o[c]) * inv * (a.norm_w ? a.norm_w[h * a.vdim + c] : 1.0f) * gate_out(a, g[c]));
}

template <typename K>
int launch_cluster(qb_ctx *ctx, K kernel, const QbRecurrence &a, uint32_t vc, size_t smem, const char *name) {
    const uint32_t split = (a.vdim + vc - 1) / vc;
    QB_REQUIRE(smem <= 220 * 1024, "linear recurrence: head of %u x %u does not fit", a.dim, a.vdim);
    QB_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(split, a.H, a.ns);
    cfg.blockDim = dim3(RT);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = ctx->stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = split; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 2;
    QB_CUDA(cudaLaunchKernelEx(&cfg, kernel, a, vc));
    QB_LAUNCHED(ctx, name);
    return QB_OK;
}

template <typename T, bool GATED>
int launch_step(qb_ctx *ctx, const QbRecurrence &a) {
    if (a.R == 1 && a.vdim % 4 == 0 && a.dim % 2 == 0 && (a.H * a.dim) % 2 == 0 && a.stride % 4 == 0 && a.state_stride % 4 == 0) {
        // slices of 32 columns spread a few heads over the SMs; with many (sequence, head) pairs a CTA takes 128
        const uint32_t vc = (uint64_t)a.ns * a.H >= 2u * (uint32_t)ctx->sm_count && a.vdim > 32 ? 128 : 32;
        const uint32_t ni = (a.dim + RT / (vc / 4) - 1) / (RT / (vc / 4)), split = (a.vdim + vc - 1) / vc;
        const size_t smem = ((size_t)2 * a.dim + (RT / 32) * vc) * sizeof(float);
        if (split <= 8 && ni <= 16) {
            if (ni <= 2) return launch_cluster(ctx, recurrence_decode_kernel<T, 2, GATED>, a, vc, smem, GATED ? "gated_recurrence_decode_kernel" : "recurrence_decode_kernel");
            if (ni <= 4) return launch_cluster(ctx, recurrence_decode_kernel<T, 4, GATED>, a, vc, smem, GATED ? "gated_recurrence_decode_kernel" : "recurrence_decode_kernel");
            if (ni <= 8) return launch_cluster(ctx, recurrence_decode_kernel<T, 8, GATED>, a, vc, smem, GATED ? "gated_recurrence_decode_kernel" : "recurrence_decode_kernel");
            return launch_cluster(ctx, recurrence_decode_kernel<T, 16, GATED>, a, vc, smem, GATED ? "gated_recurrence_decode_kernel" : "recurrence_decode_kernel");
        }
    }
    uint32_t vc = VCH;
    while ((a.vdim + vc - 1) / vc > 8) vc += VCH;
    return launch_cluster(ctx, recurrence_step_kernel<T, GATED>, a, vc, ((size_t)a.dim * vc + 3 * a.dim + a.rot.dims + (RT / 32) * vc) * sizeof(float),
                          GATED ? "gated_recurrence_step_kernel" : "recurrence_step_kernel");
}

template <bool GATED>
int launch(qb_ctx *ctx, const QbRecurrence &a) {
    const uint32_t dimr = (a.dim + 3) & ~3u;
    const size_t smem = ((size_t)2 * C * (dimr + 4) + C * VCH + (size_t)dimr * VCH + C * (C + 4) + C + 4 + dimr) * sizeof(float);
    if (a.R < 16 || (smem > 220 * 1024 && !qb_recurrence_mma_supports(a))) return a.out.f32 ? launch_step<float, GATED>(ctx, a) : launch_step<__nv_bfloat16, GATED>(ctx, a);
    if (a.S > 1 || a.rot.dims) {
        QB_CUDA(qb_launch_pdl(ctx->stream, recurrence_rotate_kernel, dim3(a.ns * a.R), dim3(RT), (size_t)(a.rot.dims * sizeof(float)), a));
        QB_LAUNCHED(ctx, GATED ? "gated_recurrence_rotate_kernel" : "recurrence_rotate_kernel");
    }
    if (qb_recurrence_mma_supports(a)) {
        QB_TRY(qb_launch_recurrence_mma(ctx, a));
    } else {
        QB_CUDA(cudaFuncSetAttribute(recurrence_chunk_kernel<GATED>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        QB_CUDA(qb_launch_pdl(ctx->stream, recurrence_chunk_kernel<GATED>, dim3(qb_recurrence_slices(a.vdim), a.H, a.ns), dim3(RT), smem, a, dimr));
        QB_LAUNCHED(ctx, GATED ? "gated_recurrence_chunk_kernel" : "recurrence_chunk_kernel");
    }
    const dim3 grid((a.ns * a.R * a.H + RT / 32 - 1) / (RT / 32));
    if (a.out.f32) QB_CUDA(qb_launch_pdl(ctx->stream, recurrence_gate_kernel<float, GATED>, grid, dim3(RT), (size_t)0, a));
    else QB_CUDA(qb_launch_pdl(ctx->stream, recurrence_gate_kernel<__nv_bfloat16, GATED>, grid, dim3(RT), (size_t)0, a));
    QB_LAUNCHED(ctx, GATED ? "gated_recurrence_gate_kernel" : "recurrence_gate_kernel");
    return QB_OK;
}

}  // namespace

int qb_launch_recurrence(qb_ctx *ctx, const QbRecurrence &a) {
    QB_REQUIRE(a.ns > 0 && a.R > 0 && a.rot.dims <= a.dim && a.stride >= 2 * a.H * (a.dim + a.vdim) + (a.gated ? 2 * a.H : 0) &&
                   a.state_stride >= qb_recurrence_state(a.H, a.dim, a.vdim, a.gated) && (a.gated ? a.row_aux && a.i_bias && a.f_bias : a.powers != nullptr),
               "linear recurrence: bad arguments");
    return a.gated ? launch<true>(ctx, a) : launch<false>(ctx, a);
}
