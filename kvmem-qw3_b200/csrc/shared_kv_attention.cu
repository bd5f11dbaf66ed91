// Grouped-query attention whose values are the key projections: query and key norm per head, rotation of a part of the head,
// a sink of score 0, one output gate per head.
//
// The values are the keys before norm and rotation, so one cached vector per token and key/value head serves both products,
// the way a latent does: with k the projection, r its root mean square and w the norm's weight, the normalised key is
// w k / r.  Dimensions that the rotation passes contribute (w q) . k / r to the score, rotated ones rot(q) . rot(w k) / r; the
// cache holds [k | rot(w k)], the factor 1 / r stands beside it in fp32 and multiplies the score.  A head of 128 with 32
// rotated dimensions is 160 numbers per token where keys and values apart are 256.
//
// Three launches: shared_kv_prepare_kernel (norms, rotation, append), the spans over the cached vectors (the kernels of absorbed
// latent attention with a group per key/value head: tcgen05 in bfloat16, fp32 arithmetic otherwise), shared_kv_merge_kernel
// (spans, sink, gate).  Many prompt rows in bfloat16: shared_kv_prefill_kernel instead of the last two.  Scores, weights and their sums are fp32.
#include "layered.h"

namespace {

constexpr int ST = 256;

// A warp per head: blocks of (rows, 8 heads); heads past H are key heads.
template <typename T>
__global__ void __launch_bounds__(ST)
shared_kv_prepare_kernel(QbSharedKv a) {
    QB_PDL_ENTER();
    extern __shared__ float sm[];
    const QbLatent &L = a.at;
    const uint32_t m = blockIdx.x, s = m / L.R, r = m % L.R, tid = threadIdx.x, w = tid >> 5, lane = tid & 31;
    const uint32_t dim = L.rank, dims = L.rot.dims, half = dims / 2, G = L.groups, hg = L.heads_per_group(), P = L.pitch(), rp = L.rankp();
    float *cs = sm, *sn = cs + half, *vec = sn + half + w * dim;
    const int pos = L.seq_pos[s] + (int)r;
    for (uint32_t i = tid; i < half; i += ST) qb_rot_angle(L.rot, pos, i, cs[i], sn[i]);
    __syncthreads();
    const uint32_t head = blockIdx.y * (ST / 32) + w;
    if (head >= L.H + G) return;
    const bool is_k = head >= L.H;
    const size_t base = (size_t)m * a.stride + (size_t)head * dim, ps = (size_t)L.ns * L.R * a.stride;
    float ss = 0.0f;
    for (uint32_t i = lane; i < dim; i += 32) {
        const float v = qb_sum8(a.proj, base + i, a.S, ps);
        vec[i] = v;
        ss += v * v;
    }
    const float inv = rsqrtf(warp_sum(ss) / (float)dim + L.eps);
    __syncwarp();
    const float *wn = is_k ? a.k_norm : a.q_norm;
    const float f = is_k ? 1.0f : inv;                       // a key's 1 / r stays outside
    auto rotated = [&](uint32_t j) -> float {
        uint32_t i, p; bool first;
        qb_rot_pair(L.rot, j, i, p, first);
        const float u = vec[j] * f * wn[j], v = vec[p] * f * wn[p];
        return first ? u * cs[i] - v * sn[i] : u * cs[i] + v * sn[i];
    };
    T *dst;
    if (is_k) {
        const uint32_t g = head - L.H;
        const int64_t at = qb_latent_slot(L, L.page_table + (size_t)s * L.pt_stride, (uint32_t)pos);
        if (at < 0) {
            if (lane == 0) atomicExch(L.err_flag, 3002);     // an unassigned page: nothing is appended
            return;
        }
        dst = (T *)L.cache + ((size_t)at * G + g) * P;
        if (lane == 0) a.key_scale[(size_t)at * G + g] = inv;
    } else {
        dst = (T *)L.qa + ((((size_t)s * G + head / hg) * L.R + r) * hg + head % hg) * P;
    }
    for (uint32_t i = lane; i < P; i += 32) {
        float v = 0.0f;
        if (i >= rp) { if (i - rp < dims) v = rotated(i - rp); }
        else if (i < dim) v = is_k ? vec[i] : i < dims ? 0.0f : vec[i] * inv * wn[i] * a.k_norm[i];
        dst[i] = qb_cast<T>(v);
    }
}

// What the merge of (row m, head h) reads: its spans, how many of them are visible, the sink's share and the gate.
struct Merge { const float *ml, *acc; uint32_t n; float mx, factor; };
__device__ __forceinline__ Merge merge_of(const QbSharedKv &a, uint32_t m, uint32_t h, uint32_t n_splits, uint32_t lane) {
    const QbLatent &L = a.at;
    const uint32_t s = m / L.R, r = m % L.R, hg = L.heads_per_group(), base = (uint32_t)L.seq_pos[s];
    const size_t q = (((size_t)s * L.groups + h / hg) * L.R + r) * hg + h % hg;
    const float g = qb_sum8(a.proj, (size_t)m * a.stride + (size_t)(L.H + L.groups) * L.rank + h, a.S, (size_t)L.ns * L.R * a.stride);
    Merge o;
    o.ml = L.part_ml + q * n_splits * 2;
    o.acc = L.part_acc + q * n_splits * L.rank;
    o.n = min((base + r) / qb_latent_span(base + L.R, L.max_splits) + 1, n_splits);
    o.mx = 0.0f;                                              // the sink's score
    for (uint32_t i = lane; i < o.n; i += 32) o.mx = fmaxf(o.mx, o.ml[2 * i]);
    o.mx = warp_max(o.mx);
    float den = 0.0f;
    for (uint32_t i = lane; i < o.n; i += 32) den += o.ml[2 * i + 1] * expf(o.ml[2 * i] - o.mx);
    o.factor = qb_sigmoid(g) / (warp_sum(den) + expf(-o.mx));
    return o;
}

// Few spans: a warp per (row, head).
template <typename T>
__global__ void __launch_bounds__(ST)
shared_kv_merge_kernel(QbSharedKv a, uint32_t n_splits) {
    QB_PDL_ENTER();
    const QbLatent &L = a.at;
    const uint32_t t = blockIdx.x * (ST / 32) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (t >= L.ns * L.R * L.H) return;
    const uint32_t m = t / L.H, h = t % L.H;
    const Merge o = merge_of(a, m, h, n_splits, lane);
    T *out = (T *)L.out.p + (size_t)m * L.out.ld + (size_t)h * L.rank;
    for (uint32_t c = lane; c < L.rank; c += 32) {
        float v = 0.0f;
#pragma unroll 4
        for (uint32_t i = 0; i < o.n; ++i) v = fmaf(expf(o.ml[2 * i] - o.mx), o.acc[(size_t)i * L.rank + c], v);
        out[c] = qb_cast<T>(v * o.factor);
    }
}
// Many spans: a CTA per (row, head), its warps take spans by turns, 128 columns at a time.
template <typename T>
__global__ void __launch_bounds__(ST)
shared_kv_merge_wide_kernel(QbSharedKv a, uint32_t n_splits) {
    QB_PDL_ENTER();
    __shared__ float part[ST / 32][128];
    const QbLatent &L = a.at;
    const uint32_t m = blockIdx.x / L.H, h = blockIdx.x % L.H, w = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const Merge o = merge_of(a, m, h, n_splits, lane);
    T *out = (T *)L.out.p + (size_t)m * L.out.ld + (size_t)h * L.rank;
    for (uint32_t c0 = 0; c0 < L.rank; c0 += 128) {
        float v[4] = {};
#pragma unroll 4
        for (uint32_t i = w; i < o.n; i += ST / 32) {
            const float e = expf(o.ml[2 * i] - o.mx), *acc = o.acc + (size_t)i * L.rank + c0 + lane;
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (c0 + lane + 32 * j < L.rank) v[j] = fmaf(e, acc[32 * j], v[j]);
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) part[w][lane + 32 * j] = v[j];
        __syncthreads();
        const uint32_t c = threadIdx.x;
        if (c < 128 && c0 + c < L.rank) {
            float t = 0.0f;
#pragma unroll
            for (int i = 0; i < ST / 32; ++i) t += part[i][c];
            out[c0 + c] = qb_cast<T>(t * o.factor);
        }
        __syncthreads();
    }
}

template <typename T>
int launch_merge(qb_ctx *ctx, const QbSharedKv &a, uint32_t n_splits) {
    const uint32_t n = a.at.ns * a.at.R * a.at.H;
    if (n_splits > 4) QB_CUDA(qb_launch_pdl(ctx->stream, shared_kv_merge_wide_kernel<T>, dim3(n), dim3(ST), (size_t)0, a, n_splits));
    else QB_CUDA(qb_launch_pdl(ctx->stream, shared_kv_merge_kernel<T>, dim3((n + ST / 32 - 1) / (ST / 32)), dim3(ST), (size_t)0, a, n_splits));
    QB_LAUNCHED(ctx, "shared_kv_merge_kernel");
    return QB_OK;
}

// Queries a span kernel's CTA takes at most (what fills the GPU is counted in these).
constexpr uint32_t SPAN_QUERIES = 48, MAX_SPANS = 64, CTAS_PER_SM = 6;

}  // namespace

// Spans per sequence that fill the GPU about twice over with the CTAs that small tiles leave room for on an SM.
uint32_t qb_shared_kv_max_splits(const QbLatent &a, uint32_t ns, uint32_t R, uint32_t sms) {
    const uint64_t ctas = (uint64_t)ns * a.groups * ((R * a.heads_per_group() + SPAN_QUERIES - 1) / SPAN_QUERIES);
    return (uint32_t)std::max<uint64_t>(1, std::min<uint64_t>(MAX_SPANS, (uint64_t)CTAS_PER_SM * sms / ctas));
}
size_t qb_shared_kv_part_floats(const QbLatent &a, uint32_t rows_cap, uint32_t n_seqs, uint32_t sms) {
    // (queries x spans): at most one span per query, or CTAs x queries of a CTA
    const size_t many = (size_t)std::max(rows_cap, n_seqs) * a.H, few = (size_t)CTAS_PER_SM * sms * SPAN_QUERIES;
    return std::max(many, few) * a.rank;
}

int qb_launch_shared_kv(qb_ctx *ctx, const QbSharedKv &args) {
    QbSharedKv a = args;
    QbLatent &L = a.at;
    L.err_flag = ctx->err_flag_dev;
    L.key_scale = a.key_scale;
    const uint32_t rows = L.ns * L.R, heads = L.H + L.groups;
    QB_REQUIRE(rows > 0 && L.groups > 0 && L.H % L.groups == 0 && L.rot.dims <= L.rank && L.rot.dims % 2 == 0 && L.rot.dims == L.rot_dim &&
                   a.stride >= heads * L.rank + L.H, "shared key/value attention: bad arguments");
    const size_t smem = ((size_t)L.rot.dims + (ST / 32) * L.rank) * sizeof(float);
    QB_REQUIRE(smem <= 48 * 1024, "shared key/value attention: heads of %u do not fit", L.rank);
    const dim3 grid(rows, (heads + ST / 32 - 1) / (ST / 32));
    if (L.f32) QB_CUDA(qb_launch_pdl(ctx->stream, shared_kv_prepare_kernel<float>, grid, dim3(ST), smem, a));
    else QB_CUDA(qb_launch_pdl(ctx->stream, shared_kv_prepare_kernel<__nv_bfloat16>, grid, dim3(ST), smem, a));
    QB_LAUNCHED(ctx, "shared_kv_prepare_kernel");
    if (qb_shared_kv_prefill_supports(L, (uint32_t)ctx->sm_count)) return qb_launch_shared_kv_prefill(ctx, a);
    const uint32_t n_splits = std::min(L.max_splits, (L.max_pos + 63) / 64);
    if (qb_latent_tc_supports(L)) QB_TRY(qb_launch_latent_split_tc(ctx, L, n_splits));
    else QB_TRY(qb_launch_latent_split_simt(ctx, L, n_splits));
    return L.f32 ? launch_merge<float>(ctx, a, n_splits) : launch_merge<__nv_bfloat16>(ctx, a, n_splits);
}
