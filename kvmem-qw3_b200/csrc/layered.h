// Layered models: decoders described layer by layer in a config.json (mixer type and sizes, feed-forward, an optional loop
// over a span of layers, layers that share weights), with dense bfloat16 weights.  Mechanisms (linear_recurrence.cu,
// latent_attention.cu, shared_kv_attention.cu, dense_gemm.cu, layered_norm.cu) take their constants as arguments;
// layered_model.cu composes them.
#pragma once

#include "dense_gemm.h"

// A rotary embedding on the device: pair i of the first `dims` dimensions turns by position * freq[i]; cos and sin are
// multiplied by amp.  interleaved: pairs (2i, 2i + 1), else (i, i + dims / 2).
struct QbRotary {
    const float *freq = nullptr;
    float amp = 1.0f;
    uint32_t dims = 0;
    bool interleaved = false;
};

#ifdef __CUDACC__
template <typename T> __device__ __forceinline__ T qb_cast(float v);
template <> __device__ __forceinline__ float qb_cast<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 qb_cast<__nv_bfloat16>(float v) { return __float2bfloat16(v); }
__device__ __forceinline__ float qb_f32(float v) { return v; }
__device__ __forceinline__ float qb_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float qb_sigmoid(float z) { return __fdiv_rn(1.0f, 1.0f + expf(-z)); }
// 32-bit angles: cos and sin of pair i at a position
__device__ __forceinline__ void qb_rot_angle(const QbRotary &r, int pos, uint32_t i, float &c, float &s) {
    sincosf((float)pos * r.freq[i], &s, &c);
    c *= r.amp;
    s *= r.amp;
}
// element j of a rotated vector: its pair index, its partner, and whether it is the first of the pair
__device__ __forceinline__ void qb_rot_pair(const QbRotary &r, uint32_t j, uint32_t &i, uint32_t &partner, bool &first) {
    if (r.interleaved) { i = j >> 1; partner = j ^ 1; first = !(j & 1); }
    else { const uint32_t h = r.dims / 2; first = j < h; i = first ? j : j - h; partner = first ? j + h : j - h; }
}
// Sum of up to 8 K-segment partials of one product, ascending, with every load in flight.
__device__ __forceinline__ float qb_sum8(const float *p, size_t idx, uint32_t S, size_t pstride) {
    if (S == 1) return p[idx];
    float v[8];
#pragma unroll
    for (uint32_t s = 0; s < 8; ++s) v[s] = s < S ? p[idx + s * pstride] : 0.0f;
    float t = v[0];
#pragma unroll
    for (uint32_t s = 1; s < 8; ++s) t += v[s];
    return t;
}
// Sum over a block of `nwarps` warps; every thread returns it.  red: nwarps floats of shared memory.
__device__ __forceinline__ float qb_block_sum(float v, float *red, uint32_t nwarps) {
    v = warp_sum(v);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.0f;
    for (uint32_t i = 0; i < nwarps; ++i) t += red[i];
    return t;
}
#endif

// ---- residual, loop additions and norm in one launch (layered_norm.cu) ------------------------------------------------
struct QbLayerNorm {
    uint32_t M = 0, n = 0;
    float eps = 0.0f;
    bool center = false;                      // layer norms (mean off first), else RMS norms
    float *x = nullptr;                       // residual stream [M][n]
    // source of the row: an embedding row (scaled; normalised with embed_w where given), or x + sum of parts (the sum normalised
    // with post_w where given)
    const int32_t *tokens = nullptr;
    const __nv_bfloat16 *embed = nullptr;     // [vocab][n]
    const float *embed_w = nullptr;
    float embed_scale = 1.0f;
    uint32_t vocab = 0;
    const float *parts = nullptr;             // [S][M][n]
    uint32_t S = 0;
    const float *row_ss = nullptr;            // sums of squares [M][ss_n] of ss_len elements: the sum of parts is divided by their
    uint32_t ss_n = 0, ss_len = 0;            // root mean square first (a norm that commutes with the product)
    const float *post_w = nullptr;            // norm on the sublayer's result, gain [n]
    const int32_t *row_map = nullptr;         // source rows of x (the stream is not written then), below x_rows
    uint32_t x_rows = 0;
    int *err_flag = nullptr;
    float *trace = nullptr;                   // copy of the residual before the loop's additions [M][n]
    float *emb_store = nullptr;               // the embedding output is kept here [M][n]
    const float *emb_add = nullptr;           // ... and added
    const float *step = nullptr;              // vector [n] added to every row
    const float *w = nullptr;                 // gain of the norm that follows; null: the row goes out as it is
    QbActBuf out;
};
int qb_launch_layer_norm(qb_ctx *ctx, const QbLayerNorm &a);

// ---- linear recurrences (linear_recurrence.cu) ---------------------------------------------------------------------------
// A matrix state per head, S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, normalised and gated.  Rows are grouped per
// sequence (R rows each, consecutive positions).
static const uint32_t QB_REC_CHUNK = 64, QB_REC_SLICE = 32;
struct QbRecurrence {
    float *proj = nullptr;                    // [S][rows][stride]: q (H*dim) | k (H*dim) | v (H*vdim) | g (H*vdim) | gated: i (H) | f (H)
    uint32_t S = 1, stride = 0;
    uint32_t ns = 0, R = 0, H = 0, dim = 0, vdim = 0;
    float eps = 0.0f;
    QbRotary rot;                             // of q and k
    bool act = false;                         // silu on q, k and v
    float qscale = 1.0f, kscale = 1.0f;
    bool sigmoid_gate = false;                // the output's gate: sigmoid(g), else silu(g)
    const float *norm_w = nullptr;            // [H*vdim] weight of the output's norm, or none
    // The output's norm is per head, or (row_ss set) spans all heads: the rows go out without it, and their sums of squares
    // [rows][H] go to the consumer of the output projection, which scales its rows.
    float *row_ss = nullptr;
    const float *powers = nullptr;            // fixed decays: [H][QB_REC_CHUNK + 1]: decay^0 .. decay^64
    // gated: log gates cap * tanh((z + bias) / cap) per token and head (the forget gate through a log sigmoid), running maximum,
    // normaliser
    bool gated = false;
    const float *i_bias = nullptr, *f_bias = nullptr;
    float cap = 1.0f;
    float *row_aux = nullptr;                 // scratch [rows][H][2]
    const int32_t *seq_pos = nullptr;
    float *state = nullptr;                   // [ns][state_stride]
    size_t state_stride = 0;
    QbActBuf out;                             // [rows][H*vdim]
};
__host__ __device__ inline uint32_t qb_recurrence_slices(uint32_t vdim) { return (vdim + QB_REC_SLICE - 1) / QB_REC_SLICE; }
// Floats of one sequence's state: [H][dim][vdim]; gated: also n [H][dim] and m [H][slices].
inline size_t qb_recurrence_state(uint32_t H, uint32_t dim, uint32_t vdim, bool gated) {
    const size_t n = (size_t)H * dim * vdim + (gated ? (size_t)H * (dim + qb_recurrence_slices(vdim)) : 0);
    return (n + 3) & ~(size_t)3;
}
int qb_launch_recurrence(qb_ctx *ctx, const QbRecurrence &a);
// The blocks of a prompt chunk on the tensor cores (linear_recurrence_mma.cu): bfloat16 models, heads up to 256.
bool qb_recurrence_mma_supports(const QbRecurrence &a);
int qb_launch_recurrence_mma(qb_ctx *ctx, const QbRecurrence &a);

// ---- latent attention (latent_attention.cu) ----------------------------------------------------------------------------
// Keys and values of all heads come from one latent vector per token; the cache holds the latent and one rotated key part
// shared by the heads.  Few rows: the key projection is absorbed into the query and attention runs over the latents
// themselves.  Prompt chunks: keys and values are expanded head by head first.
struct QbLatent {
    const float *proj = nullptr;              // [S][rows][stride]: q (H*(dim+rot_dim)) | latent (rank) | shared key part (rot_dim)
    uint32_t S = 1, stride = 0;
    uint32_t ns = 0, R = 0, H = 0, dim = 0, rot_dim = 0, vdim = 0, rank = 0;
    float eps = 0.0f, scale = 1.0f;
    QbRotary rot;
    const float *norm_w = nullptr, *sink = nullptr;      // [rank], [H]
    const QbDense *ukv = nullptr;             // per head: dimp key rows, then vdimp value rows (rows past dim / vdim are zero)
    const int32_t *seq_pos = nullptr, *page_table = nullptr;
    uint32_t pt_stride = 0, page_size = 0, max_pos = 0;
    void *cache = nullptr;                    // [slots][groups][rankp + rotp], activation type
    // Key/value groups: `groups` cached vectors per token, each attended by H / groups consecutive heads (latent attention: one,
    // by all); key_scale [slots][groups]: a factor of a vector's scores.  Queries qa and spans lie group by group:
    // [sequence][group][row][head of the group].
    uint32_t groups = 1;
    const float *key_scale = nullptr;
    uint64_t slots = 0;
    bool ingest = false;                      // a prompt chunk of one sequence
    uint32_t max_splits = 1;                  // spans a sequence's keys are cut into at most (absorbed form)
    // scratch (sizes: QbLatentScratch)
    void *q = nullptr, *qa = nullptr;
    float *part_acc = nullptr, *part_ml = nullptr;
    QbActBuf lat;
    __nv_bfloat16 *kr = nullptr, *kv = nullptr;
    QbActBuf out;                             // [rows][H*vdim]
    bool f32 = false;
    int *err_flag = nullptr;
    __host__ __device__ uint32_t dimp() const { return (dim + 15) & ~15u; }
    __host__ __device__ uint32_t rotp() const { return (rot_dim + 15) & ~15u; }
    __host__ __device__ uint32_t vdimp() const { return (vdim + 15) & ~15u; }
    __host__ __device__ uint32_t rankp() const { return (rank + 15) & ~15u; }
    __host__ __device__ uint32_t pitch() const { return rankp() + rotp(); }
    __host__ __device__ uint32_t heads_per_group() const { return H / groups; }
    __host__ __device__ uint32_t group_queries() const { return R * heads_per_group(); }
};
static const uint32_t QB_LAT_ABSORB_ROWS = 16;     // rows per sequence up to which the absorbed form runs
#ifdef __CUDACC__
// Keys per span of a sequence's absorbed attention: its keys over at most max_splits spans of whole 64-key tiles.  A function
// of the sequence's own length and of how many sequences share the launch; where the cuts fall changes rounding only.
__device__ __forceinline__ uint32_t qb_latent_span(uint32_t keys, uint32_t max_splits) { return ((keys + max_splits - 1) / max_splits + 63) & ~63u; }
#endif
#ifdef __CUDACC__
// Physical slot of a key of a sequence whose page-table row is pt, or -1 (an index past the row, an unassigned page).
__device__ __forceinline__ int64_t qb_latent_slot(const QbLatent &a, const int32_t *pt, uint32_t key) {
    const uint32_t i = key / a.page_size;
    const int32_t page = i < a.pt_stride ? pt[i] : -1;
    const int64_t slot = (int64_t)page * a.page_size + key % a.page_size;
    return page >= 0 && (uint64_t)slot < a.slots ? slot : -1;
}
#endif
// Whether prompt chunks of this shape expand keys and values (bfloat16, sizes within the kernel's registers).
bool qb_latent_expands(const QbLatent &a);
// The absorbed form's spans on tcgen05 (latent_attention_tc.cu): bfloat16, 16-key pages, a latent of at most 512.
bool qb_latent_tc_supports(const QbLatent &a);
int qb_launch_latent_split_tc(qb_ctx *ctx, const QbLatent &a, uint32_t n_splits);
// ... and in fp32 arithmetic, for every shape and both types (latent_attention.cu).
int qb_launch_latent_split_simt(qb_ctx *ctx, const QbLatent &a, uint32_t n_splits);
// Spans per sequence that fill the GPU once with ns sequences in the launch.
uint32_t qb_latent_max_splits(const QbLatent &a, uint32_t ns, uint32_t sms);
// Floats of part_acc for up to rows_cap prompt rows / n_seqs decode rows.
size_t qb_latent_part_floats(const QbLatent &a, uint32_t rows_cap, uint32_t n_seqs, uint32_t sms);
int qb_launch_latent(qb_ctx *ctx, const QbLatent &a);

// ---- attention whose values are its keys (shared_kv_attention.cu) --------------------------------------------------------
// Grouped-query attention with values that are the key projections themselves.  Per head, queries and keys are divided by
// their root mean square, weighted and rotated; the softmax has a sink of score 0 without a value; each head's output has
// a gate.  The cache keeps one vector per token and key/value head, and attention runs over it like absorbed latent attention:
//     cached [k | rot(w k)]    query [0 .. 0 | w_k q_pass | rot(q)]    score = scale / rms(k) * (query . cached)
// (the dimensions that a rotation passes need the projection only, the rotated ones are kept a second time).
struct QbSharedKv {
    QbLatent at;                              // rank = head size, rot_dim = rot.dims, groups = key/value heads, key_scale, buffers
    const float *proj = nullptr;              // [S][rows][stride]: q (H*dim) | k (groups*dim) | g (H)
    uint32_t S = 1, stride = 0;
    const float *q_norm = nullptr, *k_norm = nullptr;      // [dim]
    float *key_scale = nullptr;               // [slots][groups]
};
uint32_t qb_shared_kv_max_splits(const QbLatent &a, uint32_t ns, uint32_t R, uint32_t sms);
size_t qb_shared_kv_part_floats(const QbLatent &a, uint32_t rows_cap, uint32_t n_seqs, uint32_t sms);
// Many prompt rows in one pass over the keys, up to the gated output (shared_kv_prefill_tc.cu): bfloat16, 16-key pages.
bool qb_shared_kv_prefill_supports(const QbLatent &a, uint32_t sms);
int qb_launch_shared_kv_prefill(qb_ctx *ctx, const QbSharedKv &a);
int qb_launch_shared_kv(qb_ctx *ctx, const QbSharedKv &a);
