// Device helpers shared by the linear-recurrence kernels: activations, gates, state layout.
#pragma once

#include "layered.h"

namespace qbrec {

constexpr uint32_t C = QB_REC_CHUNK, VCH = QB_REC_SLICE;

__device__ __forceinline__ float act_in(const QbRecurrence &a, float v) { return a.act ? qb_swiglu(v, 1.0f) : v; }
__device__ __forceinline__ float gate_out(const QbRecurrence &a, float g) { return a.sigmoid_gate ? qb_sigmoid(g) : qb_swiglu(g, 1.0f); }
// Log gates of head h from the two projections of a row.
__device__ __forceinline__ float log_input_gate(const QbRecurrence &a, uint32_t h, float z) { return a.cap * tanhf((z + a.i_bias[h]) / a.cap); }
__device__ __forceinline__ float log_forget_gate(const QbRecurrence &a, uint32_t h, float z) {
    const float c = a.cap * tanhf((z + a.f_bias[h]) / a.cap);
    return fminf(c, 0.0f) - log1pf(expf(-fabsf(c)));
}
__device__ __forceinline__ float normaliser(float nq, float m) { return fmaxf(fabsf(nq), expf(-m)) + 1e-6f; }
// A gated sequence state: [H][dim][vdim], then n [H][dim], then m [H][slices] (a copy per slice of a prompt chunk's CTAs).
__device__ __forceinline__ float *state_of(const QbRecurrence &a, uint32_t s) { return a.state + (size_t)s * a.state_stride; }
__device__ __forceinline__ float *state_n(const QbRecurrence &a, uint32_t s, uint32_t h) { return state_of(a, s) + (size_t)a.H * a.dim * a.vdim + (size_t)h * a.dim; }
__device__ __forceinline__ float *state_m(const QbRecurrence &a, uint32_t s, uint32_t h) {
    return state_of(a, s) + (size_t)a.H * a.dim * (a.vdim + 1) + (size_t)h * qb_recurrence_slices(a.vdim);
}
// One token's gates: decay of the state, weight of the new outer product, and the running maximum moved on.
struct StepGates { float keep, add, m; };
__device__ __forceinline__ StepGates step_gates(const QbRecurrence &a, uint32_t h, size_t base, size_t ps, float m) {
    const uint32_t ib = 2 * a.H * (a.dim + a.vdim);
    const float i = log_input_gate(a, h, qb_sum8(a.proj, base + ib + h, a.S, ps)), f = log_forget_gate(a, h, qb_sum8(a.proj, base + ib + a.H + h, a.S, ps));
    StepGates g;
    g.m = fmaxf(f + m, i);
    g.keep = expf(f + m - g.m);
    g.add = expf(i - g.m);
    return g;
}


// A block of 64 rows' gates: sums b of the log forget gates, log input gates, running maxima m, factor of the incoming state.
// D[i][j] = exp(rowd(i) + cold(j)).
struct BlockGates {
    double b[C];
    float ig[C], m[C], rowf[C];
    __device__ __forceinline__ double rowd(uint32_t i) const { return b[i] - (double)m[i]; }
    __device__ __forceinline__ double cold(uint32_t j) const { return (double)ig[j] - b[j]; }
};
// One warp, rows 2 lane and 2 lane + 1 with their projections zi, zf: a scan of the sums, then of i_j - b_j.
__device__ __forceinline__ void block_gates(const QbRecurrence &a, uint32_t h, uint32_t lane, float m0, const float (&zi)[2], const float (&zf)[2], BlockGates &g) {
    float iv[2];
    double f[2], b[2], x[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        iv[e] = log_input_gate(a, h, zi[e]);
        f[e] = (double)log_forget_gate(a, h, zf[e]);
    }
    double run = f[0] + f[1];
    for (uint32_t off = 1; off < 32; off <<= 1) {
        const double up = __shfl_up_sync(0xffffffffu, run, off);
        if (lane >= off) run += up;
    }
    b[1] = run;
    b[0] = run - f[1];
    x[0] = (double)iv[0] - b[0];
    x[1] = fmax(x[0], (double)iv[1] - b[1]);
    double mx = x[1];
    for (uint32_t off = 1; off < 32; off <<= 1) {
        const double up = __shfl_up_sync(0xffffffffu, mx, off);
        if (lane >= off) mx = fmax(mx, up);
    }
    double before = __shfl_up_sync(0xffffffffu, mx, 1);
    before = lane ? fmax(before, (double)m0) : (double)m0;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const uint32_t r = 2 * lane + e;
        const float m = (float)(b[e] + fmax(before, x[e]));
        g.b[r] = b[e];
        g.ig[r] = iv[e];
        g.m[r] = m;
        g.rowf[r] = expf((float)((double)m0 + b[e] - (double)m));
    }
}

}  // namespace qbrec
