// Dense bfloat16 weights and the products of the layered models (dense_gemm.cu).
#pragma once

#include "qb_internal.h"

#include <cuda_bf16.h>

// ---- a bfloat16 weight in device layout -----------------------------------------------------------------------------
// The matrix [rows x cols] is cut into records of 128 rows x 64 columns (16 KB), row-tile major, each stored as the
// 128-byte-swizzled shared-memory image the tensor cores read: 16-byte piece p of row r at r*128 + ((p ^ (r & 7)) << 4).
// One pipeline stage of the GEMM is one contiguous record.  Rows and columns are padded with zeros.
static const uint32_t QB_DREC_BYTES = 16384;
struct QbDense {
    uint32_t rows = 0, cols = 0, rows_pad = 0, kc = 0;      // kc = 64-column chunks
    uint8_t *rec = nullptr;
    size_t bytes() const { return (size_t)(rows_pad / 128) * kc * QB_DREC_BYTES; }
};
// 8 consecutive weights (columns 8 * c8 ...) of a row
__host__ __device__ inline size_t qb_dense_offset(uint32_t kc, uint32_t row, uint32_t c8) {
    return ((size_t)(row >> 7) * kc + (c8 >> 3)) * QB_DREC_BYTES + (row & 127) * 128 + (((c8 & 7) ^ (row & 7)) << 4);
}
int qb_dense_alloc(qb_ctx *ctx, uint32_t rows, uint32_t cols, QbDense *out);
void qb_dense_free(QbDense *w);

// Where the rows of one tensor go inside a fused weight: source row r to row0 + (r / group) * stride + r % group.
struct QbDenseRows {
    uint32_t row0 = 0, n = 0, group = 1, stride = 1;
    __host__ __device__ uint32_t dst(uint32_t r) const { return row0 + (r / group) * stride + r % group; }
};
int qb_dense_upload(qb_ctx *ctx, QbDense *w, const QbDenseRows &rows, const uint16_t *host_bf16);
int qb_dense_fill_synth(qb_ctx *ctx, QbDense *w, const QbDenseRows &rows, uint64_t seed, uint32_t tensor_id, float amp);

// ---- activations: [cap rows][ld], bfloat16 or fp32 --------------------------------------------------------------------
struct QbActBuf {
    void *p = nullptr;
    uint32_t cap = 0, ld = 0;        // ld in elements, a multiple of 8
    bool f32 = false;
};
int qb_act_alloc(qb_ctx *ctx, QbActBuf *a, uint32_t rows, uint32_t cols, bool f32);

// Feed-forward input weight: gate and up rows interleaved in groups of 16 (32 consecutive rows = 16 gate, 16 up).
__host__ __device__ inline uint32_t qb_gate_col(uint32_t f) { return (f >> 4) * 32 + (f & 15); }

// K segments a product of M rows is cut into (1 from 65 rows on); the partial sums are added by the consumer.
uint32_t qb_dense_split(const QbDense &w, uint32_t M, bool f32, uint32_t sm_count);
// parts[s][m][n] = segment s of x W^T, fp32.
int qb_dense_gemm(qb_ctx *ctx, const QbDense &w, const QbActBuf &x, uint32_t M, float *parts, uint32_t S);
// out[m][n] = bf16(x W^T) (bfloat16 activations only).
int qb_dense_gemm_bf16(qb_ctx *ctx, const QbDense &w, const QbActBuf &x, uint32_t M, __nv_bfloat16 *out, uint32_t ld);
// out[m][f] = silu(gate) * up for the interleaved [gate; up] weight: one launch when the product needs no K segments,
// otherwise partial sums in parts and a second launch.
int qb_dense_gate_up(qb_ctx *ctx, const QbDense &w, const QbActBuf &x, uint32_t M, uint32_t F, float *parts, const QbActBuf &out);
