// Layered models: configuration, weights, per-batch buffers and the forward pass (family "layered" of the executor).
//
// A config.json lists the layers -- a mixer with its sizes and an optional dense feed-forward -- and an optional span of
// layers that runs several times with the same weights; a layer may also name an earlier or later one whose weights it uses.
// A "run" is one execution of a layer's weights; every run has a cache or state of its own.  Architectures are rows of the
// loader table in engine.cu and of DESIGNS below (what a design fixes for all its models), mixers rows of MIXERS.
#include "engine.h"
#include "json_reader.h"
#include "layered.h"
#include "safetensors_reader.h"

#include <cmath>
#include <memory>
#include <string>

// ---- description ------------------------------------------------------------------------------------------------------------
enum class MixerKind { Retention, Lightning, Mlstm, Latent, SharedKv };
inline bool is_recurrent(MixerKind k) { return k == MixerKind::Retention || k == MixerKind::Lightning || k == MixerKind::Mlstm; }
struct RotarySpec {
    uint32_t dims = 0;
    double base = 1.0;
    bool stretched = false, blended = false;     // every pair turns slower by `factor` / a blend by pair (original, fast, slow)
    double factor = 1.0, original = 1.0, fast = 1.0, slow = 1.0;
};
struct MixerSpec {
    MixerKind kind = MixerKind::Retention;
    uint32_t heads = 0, dim = 0, vdim = 0, rot_dim = 0, kv_rank = 0, kv_heads = 0;
    double scale = 1.0, gate_cap = 1.0;
    std::vector<double> decay;
    RotarySpec rot;
};
struct LayerSpec { MixerSpec mixer; uint32_t ff = 0; int weights_of = -1; };   // ff 0: no feed-forward; weights_of -1: its own
// What a design fixes for all its models.
struct Design {
    const char *architecture;
    bool center;              // layer norms without bias, else RMS norms
    bool post_norm;           // a norm on each sublayer's output (times a layer scale), none on its input
    bool embed_norm;          // the embedding is normalised, else multiplied by embedding.scale
};
const Design DESIGNS[] = {
    {"Kezilix", false, false, true},
    {"Figonex", true, true, false},
};
struct LayeredSpec {
    std::string architecture;
    const Design *design = nullptr;
    double embed_scale = 1.0;
    uint32_t vocab = 0, width = 0, loop_start = 0, loop_stop = 0, loop_times = 0;     // loop_times 0: no loop
    double eps = 0.0;
    std::vector<LayerSpec> layers;
};
struct LayerRun { uint32_t layer; int pass; bool opens; };           // pass: -1 outside the loop; opens: first of a pass

struct LayeredLayer {
    QbDense w_in, w_out, w_ukv, w_gate_up, w_down;
    const float *norm1 = nullptr, *norm2 = nullptr;       // gains (post norm: times the layer scale)
    const float *lat_norm = nullptr, *sink = nullptr, *powers = nullptr, *mix_norm = nullptr, *i_bias = nullptr, *f_bias = nullptr, *q_norm = nullptr,
                *k_norm = nullptr;
    QbRotary rot;
};
struct QbLayered {
    LayeredSpec spec;
    bool f32 = false;
    std::vector<LayerRun> runs;
    std::vector<LayeredLayer> layers;
    QbDense head;
    __nv_bfloat16 *embed = nullptr;
    const float *embed_norm = nullptr, *final_norm = nullptr, *loop_step = nullptr;
};
struct QbLayeredBatch {
    std::vector<void *> cache;                 // per run: the paged cache of an attention run
    std::vector<float *> key_scale;            // ... and its factors per key (attention whose values are its keys)
    std::vector<float *> state;                // per run: the state of a recurrent run
    float *row_aux = nullptr;                  // per row and head of a recurrent layer: sums of squares / normalisers
    QbActBuf x, mix, ff, lat;                  // normalised rows, mixer output, feed-forward hidden rows, gathered latents
    float *parts = nullptr, *emb = nullptr, *part_acc = nullptr, *part_ml = nullptr;
    void *q = nullptr, *qa = nullptr;
    __nv_bfloat16 *kr = nullptr, *kv = nullptr;
    float *trace = nullptr;                    // [runs][rows_cap][width] when enabled
    uint32_t trace_rows = 0;
};

namespace {

using qbjson::Value;

int bad(const char *what) { return qb_fail(QB_ERR_INVALID, "config.json: %s", what); }

// A positive integer member.
int need_u32(const Value &o, const char *key, uint32_t &out) {
    const Value *v = o.get(key);
    if (!v || v->kind != Value::Number || v->num < 1 || v->num > 4e9 || v->num != std::floor(v->num))
        return qb_fail(QB_ERR_INVALID, "config.json: %s must be a positive integer", key);
    out = (uint32_t)v->num;
    return QB_OK;
}
int need_num(const Value &o, const char *key, double &out) {
    const Value *v = o.get(key);
    if (!v || v->kind != Value::Number) return qb_fail(QB_ERR_INVALID, "config.json: %s must be a number", key);
    out = v->num;
    return QB_OK;
}

int parse_rotary(const Value &mixer, RotarySpec &r) {
    const Value *v = mixer.get("rot");
    if (!v || v->is_null()) return QB_OK;
    QB_TRY(need_u32(*v, "dims", r.dims));
    QB_TRY(need_num(*v, "base", r.base));
    QB_REQUIRE(r.dims % 2 == 0, "config.json: rot.dims must be even");
    const Value *s = v->get("scaling");
    if (s && !s->is_null()) {
        QB_TRY(need_num(*s, "factor", r.factor));
        r.blended = s->get("original") || s->get("fast") || s->get("slow");
        r.stretched = !r.blended;
        if (r.stretched) return QB_OK;
        QB_TRY(need_num(*s, "original", r.original));
        QB_TRY(need_num(*s, "fast", r.fast));
        QB_TRY(need_num(*s, "slow", r.slow));
    }
    return QB_OK;
}

int parse_decay(const Value &v, MixerSpec &m) {
    const Value *d = v.get("decay");
    QB_REQUIRE(d && d->items.size() == m.heads, "config.json: decay must list one number per head");
    for (const Value &x : d->items) m.decay.push_back(x.num);
    return QB_OK;
}
int parse_retention(const Value &v, MixerSpec &m) {
    m.kind = MixerKind::Retention;
    QB_TRY(parse_decay(v, m));
    QB_REQUIRE(m.rot.dims <= m.dim, "config.json: rot.dims exceeds the head");
    return QB_OK;
}
int parse_latent(const Value &v, MixerSpec &m) {
    m.kind = MixerKind::Latent;
    QB_TRY(need_u32(v, "rot_dim", m.rot_dim));
    QB_TRY(need_u32(v, "kv_rank", m.kv_rank));
    QB_TRY(need_num(v, "scale", m.scale));
    QB_REQUIRE(m.rot.dims <= m.rot_dim, "config.json: rot.dims exceeds rot_dim");
    return QB_OK;
}
int parse_lightning(const Value &v, MixerSpec &m) {
    m.kind = MixerKind::Lightning;
    return parse_decay(v, m);
}
int parse_mlstm(const Value &v, MixerSpec &m) {
    m.kind = MixerKind::Mlstm;
    QB_TRY(need_num(v, "gate_cap", m.gate_cap));
    QB_REQUIRE(m.gate_cap > 0, "config.json: gate_cap must be positive");
    return QB_OK;
}
int parse_shared_kv(const Value &v, MixerSpec &m) {
    m.kind = MixerKind::SharedKv;
    QB_TRY(need_u32(v, "kv_heads", m.kv_heads));
    QB_TRY(need_num(v, "scale", m.scale));
    QB_REQUIRE(m.heads % m.kv_heads == 0, "config.json: heads must be a multiple of kv_heads");
    QB_REQUIRE(m.vdim == m.dim, "config.json: the values are the keys, vdim must equal dim");
    QB_REQUIRE(m.rot.dims <= m.dim, "config.json: rot.dims exceeds the head");
    return QB_OK;
}
const struct { const char *type; int (*parse)(const Value &, MixerSpec &); } MIXERS[] = {
    {"lightning", parse_lightning},
    {"mlstm", parse_mlstm},
    {"attention", parse_shared_kv},
    {"retention", parse_retention},
    {"latent_attention", parse_latent},
};

int parse_spec(const std::string &text, LayeredSpec &s) {
    Value root;
    if (!qbjson::Parser(text.data(), text.size()).parse(root) || root.kind != Value::Object) return bad("not a JSON object");
    if (const Value *a = root.get("architecture")) s.architecture = a->s;
    for (const Design &d : DESIGNS)
        if (s.architecture == d.architecture) s.design = &d;
    if (!s.design) return qb_fail(QB_ERR_UNSUPPORTED, "config.json: architecture '%s' is not known", s.architecture.c_str());
    if (!s.design->embed_norm) {
        const Value *e = root.get("embedding");
        if (!e) return bad("embedding is missing");
        QB_TRY(need_num(*e, "scale", s.embed_scale));
    }
    QB_TRY(need_u32(root, "vocab", s.vocab));
    QB_TRY(need_u32(root, "width", s.width));
    const Value *norm = root.get("norm");
    if (!norm) return bad("norm is missing");
    QB_TRY(need_num(*norm, "eps", s.eps));
    const Value *layers = root.get("layers");
    if (!layers || layers->items.empty()) return bad("layers must be a list");
    for (const Value &l : layers->items) {
        LayerSpec L;
        const Value *type = l.get("type"), *mx = l.get("mixer"), *mlp = l.get("mlp");
        if (!type || !mx) return bad("a layer needs type and mixer");
        QB_TRY(need_u32(*mx, "heads", L.mixer.heads));
        QB_TRY(need_u32(*mx, "dim", L.mixer.dim));
        QB_TRY(need_u32(*mx, "vdim", L.mixer.vdim));
        QB_TRY(parse_rotary(*mx, L.mixer.rot));
        bool known = false;
        for (const auto &m : MIXERS)
            if (type->s == m.type) { known = true; QB_TRY(m.parse(*mx, L.mixer)); }
        if (!known) return qb_fail(QB_ERR_UNSUPPORTED, "config.json: mixer %s is not known", type->s.c_str());
        if (mlp && !mlp->is_null()) {
            const Value *kind = mlp->get("kind");
            if (kind && kind->s != "dense") return qb_fail(QB_ERR_UNSUPPORTED, "config.json: feed-forward %s is not known", kind->s.c_str());
            QB_TRY(need_u32(*mlp, "ff", L.ff));
        }
        const Value *of = l.get("weights_of");
        if (of && !of->is_null()) {
            if (of->kind != Value::Number || of->num < 0 || of->num >= (double)layers->items.size() || of->num != std::floor(of->num))
                return bad("weights_of must name a layer");
            L.weights_of = (int)of->num;
        }
        s.layers.push_back(std::move(L));
    }
    // a chain of weights_of ends at a layer with weights of its own, of the same shape
    for (uint32_t i = 0; i < s.layers.size(); ++i) {
        uint32_t j = i, hops = 0;
        for (; s.layers[j].weights_of >= 0 && hops <= s.layers.size(); ++hops) j = (uint32_t)s.layers[j].weights_of;
        if (hops > s.layers.size()) return bad("weights_of goes in a circle");
        const LayerSpec &a = s.layers[i], &b = s.layers[j];
        if (a.mixer.kind != b.mixer.kind || a.mixer.heads != b.mixer.heads || a.mixer.dim != b.mixer.dim || a.mixer.vdim != b.mixer.vdim || a.ff != b.ff ||
            a.mixer.kv_heads != b.mixer.kv_heads)
            return bad("a layer with weights_of must equal the layer it names");
    }
    const Value *loop = root.get("loop");
    if (loop && !loop->is_null()) {
        double a = -1, b = -1;
        QB_TRY(need_num(*loop, "start", a));
        QB_TRY(need_num(*loop, "stop", b));
        QB_TRY(need_u32(*loop, "times", s.loop_times));
        if (a < 0 || b <= a || b > (double)s.layers.size()) return bad("loop must span some of the layers");
        s.loop_start = (uint32_t)a;
        s.loop_stop = (uint32_t)b;
    }
    return QB_OK;
}

std::vector<LayerRun> list_runs(const LayeredSpec &s) {
    std::vector<LayerRun> r;                 // (.layer: the one whose weights run)
    const uint32_t n = (uint32_t)s.layers.size(), a = s.loop_times ? s.loop_start : n, b = s.loop_times ? s.loop_stop : n;
    for (uint32_t i = 0; i < a; ++i) r.push_back({i, -1, false});
    for (uint32_t t = 0; t < s.loop_times; ++t)
        for (uint32_t i = a; i < b; ++i) r.push_back({i, (int)t, i == a});
    for (uint32_t i = b; i < n; ++i) r.push_back({i, -1, false});
    for (LayerRun &run : r)
        while (s.layers[run.layer].weights_of >= 0) run.layer = (uint32_t)s.layers[run.layer].weights_of;
    return r;
}

// Frequencies and amplitude of a rotation.  Stretched: every pair turns at 1 / factor.  Blended: pair i turns at its own frequency where a dimension makes more than
// `fast` turns over the original context, at 1 / factor of it below `slow` turns, and at a blend in between.
void rotary_freqs(const RotarySpec &r, std::vector<float> &freq, float &amp) {
    freq.assign(std::max(1u, r.dims / 2), 0.0f);
    amp = 1.0f;
    double lo = 0, hi = 0;
    if (r.blended) {
        auto at = [&](double turns) { return r.dims * std::log(r.original / (2.0 * M_PI * turns)) / (2.0 * std::log(r.base)); };
        lo = std::max(std::floor(at(r.fast)), 0.0);
        hi = std::min(std::ceil(at(r.slow)), (double)r.dims - 1.0);
        amp = (float)(0.1 * std::log(r.factor) + 1.0);
    }
    for (uint32_t i = 0; i < r.dims / 2; ++i) {
        double f = std::pow(r.base, -2.0 * i / r.dims);
        if (r.stretched) f /= r.factor;
        if (r.blended) {
            const double ramp = std::min(std::max(((double)i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
            f = f / r.factor * ramp + f * (1.0 - ramp);
        }
        freq[i] = (float)f;
    }
}

// ---- weights: from a safetensors file, or seeded -------------------------------------------------------------------------------
struct Source {
    const qbst::File *file = nullptr;          // null: seeded
    uint64_t seed = 0;
    uint32_t next_id = 1;
};

float bf16_to_f32(uint16_t v) {
    const uint32_t u = (uint32_t)v << 16;
    float f;
    memcpy(&f, &u, 4);
    return f;
}

int find_tensor(const Source &src, const std::string &name, std::initializer_list<uint64_t> shape, const qbst::Tensor **out) {
    const qbst::Tensor *t = src.file->find(name);
    if (!t) return qb_fail(QB_ERR_INVALID, "model: tensor %s is missing", name.c_str());
    if (t->dtype != "BF16" || t->bytes != t->count() * 2) return qb_fail(QB_ERR_UNSUPPORTED, "model: tensor %s has type %s, expected BF16", name.c_str(), t->dtype.c_str());
    if (t->shape != std::vector<uint64_t>(shape)) return qb_fail(QB_ERR_INVALID, "model: tensor %s does not have the shape the configuration gives it", name.c_str());
    *out = t;
    return QB_OK;
}
// A matrix [rows.n][w.cols] into its rows of a fused weight.
int put_matrix(qb_ctx *ctx, Source &src, const std::string &name, QbDense *w, const QbDenseRows &rows) {
    if (!src.file) return qb_dense_fill_synth(ctx, w, rows, src.seed, src.next_id++, (float)std::sqrt(3.0 / w->cols));
    const qbst::Tensor *t = nullptr;
    QB_TRY(find_tensor(src, name, {rows.n, w->cols}, &t));
    return qb_dense_upload(ctx, w, rows, (const uint16_t *)t->data);
}
// A vector (or a small [a][b] table) widened to fp32.
int read_f32(Source &src, const std::string &name, std::initializer_list<uint64_t> shape, float dflt, std::vector<float> &v) {
    size_t n = 1;
    for (uint64_t d : shape) n *= d;
    v.assign(n, dflt);
    if (!src.file) return QB_OK;
    const qbst::Tensor *t = nullptr;
    QB_TRY(find_tensor(src, name, shape, &t));
    for (size_t i = 0; i < n; ++i) { uint16_t raw; memcpy(&raw, t->data + 2 * i, 2); v[i] = bf16_to_f32(raw); }
    return QB_OK;
}
// fp32 numbers on the device, owned by the model.
int keep_f32(qb_ctx *ctx, qb_model *m, const std::vector<float> &v, const float **out) {
    float *dev = nullptr;
    QB_TRY(qb_upload_f32(ctx, v, &dev));
    m->owned_f32.push_back(dev);
    *out = dev;
    return QB_OK;
}
int put_f32(qb_ctx *ctx, Source &src, qb_model *m, const std::string &name, std::initializer_list<uint64_t> shape, float dflt, const float **out) {
    std::vector<float> v;
    QB_TRY(read_f32(src, name, shape, dflt, v));
    return keep_f32(ctx, m, v, out);
}
// Gain of a sublayer's norm, times the layer scale where the design has one (both bfloat16: the product is exact in fp32).
int put_gain(qb_ctx *ctx, Source &src, qb_model *m, const std::string &norm, const std::string &scale, uint32_t D, const float **out) {
    std::vector<float> v, l;
    QB_TRY(read_f32(src, norm, {D}, 1.0f, v));
    if (m->layered->spec.design->post_norm) {
        QB_TRY(read_f32(src, scale, {D}, 0.5f, l));
        for (uint32_t i = 0; i < D; ++i) v[i] *= l[i];
    }
    return keep_f32(ctx, m, v, out);
}
QbDenseRows rows_at(uint32_t row0, uint32_t n) {
    QbDenseRows r;
    r.row0 = row0; r.n = n; r.group = std::max(1u, n); r.stride = r.group;
    return r;
}
QbDenseRows rows_grouped(uint32_t row0, uint32_t n, uint32_t group, uint32_t stride) {
    QbDenseRows r;
    r.row0 = row0; r.n = n; r.group = group; r.stride = stride;
    return r;
}

// The shape of an attention layer as its kernels take it (no buffers).
QbLatent latent_shape(const MixerSpec &m, bool f32) {
    QbLatent a;
    a.H = m.heads; a.dim = m.dim; a.rot_dim = m.rot_dim; a.vdim = m.vdim; a.rank = m.kv_rank; a.f32 = f32;
    if (m.kind == MixerKind::SharedKv) { a.rank = m.dim; a.rot_dim = m.rot.dims; a.groups = m.kv_heads; }
    return a;
}

// The constants of a recurrent mixer as its kernels take them (no buffers).
QbRecurrence recurrence_shape(const MixerSpec &m) {
    QbRecurrence a;
    a.H = m.heads; a.dim = m.dim; a.vdim = m.vdim;
    a.gated = m.kind == MixerKind::Mlstm;
    a.cap = (float)m.gate_cap;
    a.act = m.kind == MixerKind::Lightning;
    a.sigmoid_gate = m.kind != MixerKind::Retention;
    if (m.kind == MixerKind::Retention) a.kscale = 1.0f / sqrtf((float)m.dim);
    if (m.kind == MixerKind::Mlstm) a.qscale = 1.0f / sqrtf((float)m.dim);
    a.state_stride = qb_recurrence_state(a.H, a.dim, a.vdim, a.gated);
    return a;
}
// The projection rows of a recurrent mixer: q | k | v | g (| i | f, padded to whole 16-byte rows of fp32 sums).
uint32_t recurrence_rows(const MixerSpec &m) {
    const uint32_t n = 2 * m.heads * (m.dim + m.vdim) + (m.kind == MixerKind::Mlstm ? 2 * m.heads : 0);
    return m.kind == MixerKind::Mlstm ? (n + 3) & ~3u : n;
}

int build_layer(qb_ctx *ctx, qb_model *m, Source &src, uint32_t i) {
    QbLayered &Y = *m->layered;
    const LayerSpec &S = Y.spec.layers[i];
    const MixerSpec &mx = S.mixer;
    LayeredLayer &L = Y.layers[i];
    const uint32_t D = Y.spec.width, H = mx.heads;
    const std::string p = "l" + std::to_string(i) + ".", q = p + "mix.", f = p + "mlp.";
    if (S.weights_of >= 0) return QB_OK;
    QB_TRY(put_gain(ctx, src, m, p + "norm1", p + "ls1", D, &L.norm1));
    std::vector<float> freq;
    rotary_freqs(mx.rot, freq, L.rot.amp);
    QB_TRY(keep_f32(ctx, m, freq, &L.rot.freq));
    L.rot.dims = mx.rot.dims;
    if (is_recurrent(mx.kind)) {
        const uint32_t qk = H * mx.dim, vv = H * mx.vdim;
        QB_TRY(qb_dense_alloc(ctx, recurrence_rows(mx), D, &L.w_in));
        QB_TRY(put_matrix(ctx, src, q + "q", &L.w_in, rows_at(0, qk)));
        QB_TRY(put_matrix(ctx, src, q + "k", &L.w_in, rows_at(qk, qk)));
        QB_TRY(put_matrix(ctx, src, q + "v", &L.w_in, rows_at(2 * qk, vv)));
        QB_TRY(put_matrix(ctx, src, q + "g", &L.w_in, rows_at(2 * qk + vv, vv)));
        std::vector<float> pw;
        for (double d : mx.decay)
            for (uint32_t n = 0; n <= QB_REC_CHUNK; ++n) pw.push_back((float)std::pow(d, (double)n));
        if (!pw.empty()) QB_TRY(keep_f32(ctx, m, pw, &L.powers));
        if (mx.kind != MixerKind::Retention) QB_TRY(put_f32(ctx, src, m, q + "norm", {vv}, 1.0f, &L.mix_norm));
        if (mx.kind == MixerKind::Mlstm) {
            QB_TRY(put_matrix(ctx, src, q + "i", &L.w_in, rows_at(2 * (qk + vv), H)));
            QB_TRY(put_matrix(ctx, src, q + "f", &L.w_in, rows_at(2 * (qk + vv) + H, H)));
            QB_TRY(put_f32(ctx, src, m, q + "i.b", {H}, 0.0f, &L.i_bias));
            QB_TRY(put_f32(ctx, src, m, q + "f.b", {H}, 3.0f, &L.f_bias));
        }
    } else if (mx.kind == MixerKind::SharedKv) {
        const uint32_t qd = H * mx.dim, kd = mx.kv_heads * mx.dim;
        QB_TRY(qb_dense_alloc(ctx, qd + kd + H, D, &L.w_in));
        QB_TRY(put_matrix(ctx, src, q + "q", &L.w_in, rows_at(0, qd)));
        QB_TRY(put_matrix(ctx, src, q + "k", &L.w_in, rows_at(qd, kd)));
        QB_TRY(put_matrix(ctx, src, q + "g", &L.w_in, rows_at(qd + kd, H)));
        QB_TRY(put_f32(ctx, src, m, q + "q.norm", {mx.dim}, 1.0f, &L.q_norm));
        QB_TRY(put_f32(ctx, src, m, q + "k.norm", {mx.dim}, 1.0f, &L.k_norm));
    } else {
        L.rot.interleaved = true;
        const QbLatent a = latent_shape(mx, Y.f32);
        const uint32_t qd = H * (mx.dim + mx.rot_dim), per = a.dimp() + a.vdimp();
        QB_TRY(qb_dense_alloc(ctx, qd + mx.kv_rank + mx.rot_dim, D, &L.w_in));
        QB_TRY(put_matrix(ctx, src, q + "q", &L.w_in, rows_at(0, qd)));
        QB_TRY(put_matrix(ctx, src, q + "dkv", &L.w_in, rows_at(qd, mx.kv_rank + mx.rot_dim)));
        // per head: its key rows, then its value rows, each padded to a multiple of 16
        QB_TRY(qb_dense_alloc(ctx, H * per, mx.kv_rank, &L.w_ukv));
        QB_TRY(put_matrix(ctx, src, q + "uk", &L.w_ukv, rows_grouped(0, H * mx.dim, mx.dim, per)));
        QB_TRY(put_matrix(ctx, src, q + "uv", &L.w_ukv, rows_grouped(a.dimp(), H * mx.vdim, mx.vdim, per)));
        QB_TRY(put_f32(ctx, src, m, q + "dkv.norm", {mx.kv_rank}, 1.0f, &L.lat_norm));
        QB_TRY(put_f32(ctx, src, m, q + "sink", {H}, 0.0f, &L.sink));
    }
    QB_TRY(qb_dense_alloc(ctx, D, H * mx.vdim, &L.w_out));
    QB_TRY(put_matrix(ctx, src, q + "o", &L.w_out, rows_at(0, D)));
    m->weight_bytes += L.w_in.bytes() + L.w_out.bytes() + L.w_ukv.bytes();
    if (S.ff) {
        QB_TRY(put_gain(ctx, src, m, p + "norm2", p + "ls2", D, &L.norm2));
        QB_TRY(qb_dense_alloc(ctx, (S.ff + 15) / 16 * 32, D, &L.w_gate_up));
        QB_TRY(put_matrix(ctx, src, f + "gate", &L.w_gate_up, rows_grouped(0, S.ff, 16, 32)));
        QB_TRY(put_matrix(ctx, src, f + "up", &L.w_gate_up, rows_grouped(16, S.ff, 16, 32)));
        QB_TRY(qb_dense_alloc(ctx, D, S.ff, &L.w_down));
        QB_TRY(put_matrix(ctx, src, f + "down", &L.w_down, rows_at(0, D)));
        m->weight_bytes += L.w_gate_up.bytes() + L.w_down.bytes();
    }
    return QB_OK;
}

__global__ void synth_embed_kernel(__nv_bfloat16 *e, uint64_t n, uint64_t seed) {
    const uint64_t i = (uint64_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) e[i] = __float2bfloat16((float)(qs_rand_u32(seed, 0, i) >> 8) * (1.0f / 8388608.0f) - 1.0f);
}

int build_model(qb_ctx *ctx, qb_model *m, Source &src) {
    QbLayered &Y = *m->layered;
    const LayeredSpec &s = Y.spec;
    const uint32_t D = s.width, V = s.vocab;
    for (uint32_t i = 0; i < s.layers.size(); ++i) QB_TRY(build_layer(ctx, m, src, i));
    QB_CUDA(cudaMalloc(&Y.embed, (size_t)V * D * 2));
    if (src.file) {
        const qbst::Tensor *t = nullptr;
        QB_TRY(find_tensor(src, "embed", {V, D}, &t));
        QB_CUDA(cudaMemcpyAsync(Y.embed, t->data, t->bytes, cudaMemcpyHostToDevice, ctx->stream));
    } else {
        synth_embed_kernel<<<(unsigned)(((uint64_t)V * D + 255) / 256), 256, 0, ctx->stream>>>(Y.embed, (uint64_t)V * D, src.seed);
        QB_LAUNCHED(ctx, "synth_embed_kernel");
    }
    if (s.design->embed_norm) QB_TRY(put_f32(ctx, src, m, "embed.norm", {D}, 1.0f, &Y.embed_norm));
    if (s.loop_times) QB_TRY(put_f32(ctx, src, m, "loop.step", {s.loop_times, D}, 0.1f, &Y.loop_step));
    QB_TRY(put_f32(ctx, src, m, "final.norm", {D}, 1.0f, &Y.final_norm));
    QB_TRY(qb_dense_alloc(ctx, V, D, &Y.head));
    QB_TRY(put_matrix(ctx, src, "head", &Y.head, rows_at(0, V)));
    m->weight_bytes += Y.head.bytes() + (size_t)V * D * 2;
    QB_CUDA(cudaStreamSynchronize(ctx->stream));       // the mapped file may go away
    return QB_OK;
}

void layered_model_free(qb_ctx *, qb_model *m) {
    QbLayered *Y = m->layered;
    if (!Y) return;
    for (LayeredLayer &L : Y->layers)
        for (QbDense *w : {&L.w_in, &L.w_out, &L.w_ukv, &L.w_gate_up, &L.w_down}) qb_dense_free(w);
    qb_dense_free(&Y->head);
    if (Y->embed) cudaFree(Y->embed);
    delete Y;
    m->layered = nullptr;
}

// ---- a batch's buffers --------------------------------------------------------------------------------------------------------------
int layered_batch_alloc(qb_ctx *ctx, qb_batch *b, size_t slots) {
    const QbLayered &Y = *b->m->layered;
    const bool f32 = Y.f32;
    const size_t es = f32 ? 4 : 2;
    const uint32_t rows = b->rows_cap, D = Y.spec.width, sms = (uint32_t)ctx->sm_count;
    QbLayeredBatch *B = b->layered = new QbLayeredBatch();
    // partial sums: whole chunks unsplit, up to 64 rows in K segments
    size_t parts = 0;
    auto consider = [&](const QbDense &w) {
        if (!w.rec) return;
        for (uint32_t M : {1u, 32u, 33u, 64u}) parts = std::max(parts, (size_t)qb_dense_split(w, M, f32, sms) * std::min(rows, 64u) * w.rows);
        parts = std::max(parts, (size_t)rows * w.rows);
    };
    uint32_t mix = 1, ff = 1, max_keys = b->pages_per_seq * b->page_size;
    size_t q = 0, qa = 0, acc = 0, ml = 0, kr = 0, kv = 0, lat_ld = 0, aux = 0;
    for (uint32_t i = 0; i < Y.layers.size(); ++i) {
        const LayeredLayer &L = Y.layers[i];
        const LayerSpec &S = Y.spec.layers[i];
        consider(L.w_in); consider(L.w_out); consider(L.w_gate_up); consider(L.w_down);
        mix = std::max(mix, S.mixer.heads * S.mixer.vdim);
        ff = std::max(ff, S.ff);
        if (is_recurrent(S.mixer.kind)) {
            if (S.mixer.kind != MixerKind::Retention) aux = std::max(aux, (size_t)rows * S.mixer.heads * 2);
            continue;
        }
        const QbLatent a = latent_shape(S.mixer, f32);
        if (S.mixer.kind == MixerKind::SharedKv) {
            const size_t pf = qb_shared_kv_part_floats(a, rows, b->n_seqs, sms);
            qa = std::max(qa, (size_t)rows * a.H * a.pitch());
            acc = std::max(acc, pf);
            ml = std::max(ml, pf / a.rank * 2);
            continue;
        }
        q = std::max(q, (size_t)rows * a.H * (a.dimp() + a.rotp()));
        qa = std::max(qa, (size_t)rows * a.H * a.pitch());
        const size_t pf = qb_latent_part_floats(a, rows, b->n_seqs, sms);
        acc = std::max(acc, pf);
        ml = std::max(ml, pf / a.rank * 2);
        if (qb_latent_expands(a)) {
            lat_ld = std::max(lat_ld, (size_t)a.rankp());
            kr = std::max(kr, (size_t)max_keys * a.rotp());
            kv = std::max(kv, (size_t)max_keys * L.w_ukv.rows);
        }
    }
    QB_TRY(qb_act_alloc(ctx, &B->x, rows, D, f32));
    QB_TRY(qb_act_alloc(ctx, &B->mix, rows, mix, f32));
    QB_TRY(qb_act_alloc(ctx, &B->ff, rows, ff, f32));
    QB_CUDA(cudaMalloc(&B->parts, parts * sizeof(float)));
    QB_CUDA(cudaMalloc(&B->emb, (size_t)rows * D * sizeof(float)));
    if (aux) QB_CUDA(cudaMalloc(&B->row_aux, aux * sizeof(float)));
    if (q) QB_CUDA(cudaMalloc(&B->q, q * es));
    if (qa) {
        QB_CUDA(cudaMalloc(&B->qa, qa * es));
        QB_CUDA(cudaMalloc(&B->part_acc, acc * sizeof(float)));
        QB_CUDA(cudaMalloc(&B->part_ml, ml * sizeof(float)));
    }
    if (kv) {
        QB_TRY(qb_act_alloc(ctx, &B->lat, max_keys, (uint32_t)lat_ld, false));
        QB_CUDA(cudaMalloc(&B->kr, kr * 2));
        QB_CUDA(cudaMalloc(&B->kv, kv * 2));
    }
    B->cache.assign(Y.runs.size(), nullptr);
    B->key_scale.assign(Y.runs.size(), nullptr);
    B->state.assign(Y.runs.size(), nullptr);
    for (size_t r = 0; r < Y.runs.size(); ++r) {
        const MixerSpec &mx = Y.spec.layers[Y.runs[r].layer].mixer;
        if (!is_recurrent(mx.kind)) {
            const QbLatent a = latent_shape(mx, f32);
            const size_t bytes = slots * a.groups * a.pitch() * es;
            QB_CUDA(cudaMalloc(&B->cache[r], bytes));
            QB_CUDA(cudaMemsetAsync(B->cache[r], 0, bytes, ctx->stream));
            if (mx.kind == MixerKind::SharedKv) {
                QB_CUDA(cudaMalloc(&B->key_scale[r], slots * a.groups * sizeof(float)));
                QB_CUDA(cudaMemsetAsync(B->key_scale[r], 0, slots * a.groups * sizeof(float), ctx->stream));
            }
        } else {
            StateBlock sb;
            sb.per_seq = sb.head = recurrence_shape(mx).state_stride;
            QB_CUDA(cudaMalloc(&B->state[r], b->n_seqs * sb.per_seq * sizeof(float)));
            QB_CUDA(cudaMemsetAsync(B->state[r], 0, b->n_seqs * sb.per_seq * sizeof(float), ctx->stream));
            sb.buf[0] = B->state[r];
            b->blocks.push_back(sb);
        }
    }
    return QB_OK;
}

void layered_batch_free(qb_batch *b) {
    QbLayeredBatch *B = b->layered;
    if (!B) return;
    for (void *p : B->cache) if (p) cudaFree(p);
    for (float *p : B->state) if (p) cudaFree(p);
    for (float *p : B->key_scale) if (p) cudaFree(p);
    void *ptrs[] = {B->x.p, B->mix.p, B->ff.p, B->lat.p, B->parts, B->emb, B->part_acc, B->part_ml, B->q, B->qa, B->kr, B->kv, B->trace, B->row_aux};
    for (void *p : ptrs) if (p) cudaFree(p);
    delete B;
    b->layered = nullptr;
}

// ---- forward --------------------------------------------------------------------------------------------------------------------------
// parts = W x in K segments; returns their number.
int product(qb_ctx *ctx, QbLayeredBatch *B, const QbDense &w, const QbActBuf &x, uint32_t rows, uint32_t *S) {
    *S = qb_dense_split(w, rows, x.f32, (uint32_t)ctx->sm_count);
    return qb_dense_gemm(ctx, w, x, rows, B->parts, *S);
}

int recurrent_block(qb_ctx *ctx, qb_batch *b, uint32_t run, const RowSet &rs, uint32_t *S) {
    const QbLayered &Y = *b->m->layered;
    QbLayeredBatch *B = b->layered;
    const LayeredLayer &L = Y.layers[Y.runs[run].layer];
    const MixerSpec &mx = Y.spec.layers[Y.runs[run].layer].mixer;
    QbRecurrence a = recurrence_shape(mx);
    QB_TRY(product(ctx, B, L.w_in, B->x, rs.rows(), &a.S));
    a.proj = B->parts; a.stride = L.w_in.rows;
    a.ns = rs.ns; a.R = rs.R; a.eps = (float)Y.spec.eps;
    a.rot = L.rot; a.powers = L.powers; a.seq_pos = rs.seq_pos;
    a.norm_w = L.mix_norm; a.i_bias = L.i_bias; a.f_bias = L.f_bias;
    if (mx.kind == MixerKind::Lightning) a.row_ss = B->row_aux;
    if (a.gated) a.row_aux = B->row_aux;
    a.state = B->state[run] + (size_t)rs.seq0 * a.state_stride;
    a.out = B->mix;
    QB_TRY(qb_launch_recurrence(ctx, a));
    return product(ctx, B, L.w_out, B->mix, rs.rows(), S);
}

// Fields that the attention mixers share: rows, positions, pages, cache, span buffers.
void attention_common(const qb_batch *b, uint32_t run, const RowSet &rs, const LayeredLayer &L, const MixerSpec &mx, QbLatent &a) {
    QbLayeredBatch *B = b->layered;
    a.ns = rs.ns; a.R = rs.R; a.eps = (float)b->m->layered->spec.eps; a.scale = (float)mx.scale;
    a.rot = L.rot;
    a.seq_pos = rs.seq_pos; a.max_pos = rs.max_pos; a.ingest = rs.ingest;
    a.page_table = b->page_table + (size_t)rs.seq0 * b->pages_per_seq; a.pt_stride = b->pages_per_seq; a.page_size = b->page_size;
    a.cache = B->cache[run];
    a.slots = b->slots;
    a.qa = B->qa; a.part_acc = B->part_acc; a.part_ml = B->part_ml;
    a.out = B->mix;
}

int shared_kv_block(qb_ctx *ctx, qb_batch *b, uint32_t run, const RowSet &rs, uint32_t *S) {
    const QbLayered &Y = *b->m->layered;
    QbLayeredBatch *B = b->layered;
    const LayeredLayer &L = Y.layers[Y.runs[run].layer];
    const MixerSpec &mx = Y.spec.layers[Y.runs[run].layer].mixer;
    QbSharedKv a;
    a.at = latent_shape(mx, Y.f32);
    QB_TRY(product(ctx, B, L.w_in, B->x, rs.rows(), &a.S));
    attention_common(b, run, rs, L, mx, a.at);
    a.at.max_splits = qb_shared_kv_max_splits(a.at, rs.ns, rs.R, (uint32_t)ctx->sm_count);
    a.proj = B->parts; a.stride = L.w_in.rows;
    a.q_norm = L.q_norm; a.k_norm = L.k_norm; a.key_scale = B->key_scale[run];
    QB_TRY(qb_launch_shared_kv(ctx, a));
    return product(ctx, B, L.w_out, B->mix, rs.rows(), S);
}

int latent_block(qb_ctx *ctx, qb_batch *b, uint32_t run, const RowSet &rs, uint32_t *S) {
    const QbLayered &Y = *b->m->layered;
    QbLayeredBatch *B = b->layered;
    const LayeredLayer &L = Y.layers[Y.runs[run].layer];
    const MixerSpec &mx = Y.spec.layers[Y.runs[run].layer].mixer;
    QbLatent a = latent_shape(mx, Y.f32);
    QB_TRY(product(ctx, B, L.w_in, B->x, rs.rows(), &a.S));
    a.proj = B->parts; a.stride = L.w_in.rows;
    attention_common(b, run, rs, L, mx, a);
    a.norm_w = L.lat_norm; a.sink = L.sink; a.ukv = &L.w_ukv;
    a.max_splits = qb_latent_max_splits(a, rs.ns, (uint32_t)ctx->sm_count);
    a.q = B->q; a.lat = B->lat; a.kr = B->kr; a.kv = B->kv;
    QB_TRY(qb_launch_latent(ctx, a));
    return product(ctx, B, L.w_out, B->mix, rs.rows(), S);
}

int layered_forward(qb_ctx *ctx, qb_batch *b, const int32_t *tokens_dev, const RowSet &rs, bool checkpoints) {
    QB_REQUIRE(!checkpoints, "layered models keep no per-row state checkpoints");
    const QbLayered &Y = *b->m->layered;
    const LayeredSpec &s = Y.spec;
    QbLayeredBatch *B = b->layered;
    const uint32_t rows = rs.rows(), D = s.width, n_runs = (uint32_t)Y.runs.size();
    const Design &d = *s.design;
    auto norm_launch = [&]() {
        QbLayerNorm n;
        n.M = rows; n.n = D; n.eps = (float)s.eps; n.center = d.center; n.x = b->hid; n.out = B->x;
        return n;
    };
    // What the norm launch before run r (r = n_runs: the output norm) does for it, with what the loop adds in front of a pass.
    auto open_run = [&](QbLayerNorm &n, uint32_t r) {
        if (r == n_runs) { n.w = Y.final_norm; return; }
        const LayerRun &run = Y.runs[r];
        n.w = d.post_norm ? nullptr : Y.layers[run.layer].norm1;
        if (run.opens) {
            if (run.pass > 0) n.emb_add = B->emb;
            n.step = Y.loop_step + (size_t)run.pass * D;
        }
    };
    B->trace_rows = rows;
    {
        QbLayerNorm n = norm_launch();
        open_run(n, 0);
        n.tokens = tokens_dev; n.embed = Y.embed; n.embed_w = Y.embed_norm; n.embed_scale = (float)s.embed_scale; n.vocab = s.vocab;
        n.emb_store = s.loop_times > 1 ? B->emb : nullptr;
        QB_TRY(qb_launch_layer_norm(ctx, n));
    }
    for (uint32_t r = 0; r < n_runs; ++r) {
        const LayeredLayer &L = Y.layers[Y.runs[r].layer];
        const LayerSpec &S = s.layers[Y.runs[r].layer];
        uint32_t seg = 1;
        if (is_recurrent(S.mixer.kind)) QB_TRY(recurrent_block(ctx, b, r, rs, &seg));
        else if (S.mixer.kind == MixerKind::SharedKv) QB_TRY(shared_kv_block(ctx, b, r, rs, &seg));
        else QB_TRY(latent_block(ctx, b, r, rs, &seg));
        QbLayerNorm n = norm_launch();                       // after the mixer
        if (S.mixer.kind == MixerKind::Lightning) { n.row_ss = B->row_aux; n.ss_n = S.mixer.heads; n.ss_len = S.mixer.heads * S.mixer.vdim; }
        n.parts = B->parts; n.S = seg;
        if (d.post_norm) n.post_w = L.norm1;
        if (S.ff) {
            if (!d.post_norm) n.w = L.norm2;
            QB_TRY(qb_launch_layer_norm(ctx, n));
            QB_TRY(qb_dense_gate_up(ctx, L.w_gate_up, B->x, rows, S.ff, B->parts, B->ff));
            QB_TRY(product(ctx, B, L.w_down, B->ff, rows, &seg));
            n = norm_launch();                               // after the feed-forward
            n.parts = B->parts; n.S = seg;
            if (d.post_norm) n.post_w = L.norm2;
        }
        open_run(n, r + 1);
        if (B->trace) n.trace = B->trace + (size_t)r * b->rows_cap * D;
        QB_TRY(qb_launch_layer_norm(ctx, n));
    }
    return QB_OK;
}

int layered_head(qb_ctx *ctx, qb_batch *b, const int32_t *row_map, uint32_t rows, float *dst) {
    const QbLayered &Y = *b->m->layered;
    QbLayeredBatch *B = b->layered;
    if (row_map) {
        QbLayerNorm n;
        n.M = rows; n.n = Y.spec.width; n.eps = (float)Y.spec.eps; n.center = Y.spec.design->center; n.x = b->hid; n.x_rows = b->rows_cap + b->n_seqs; n.row_map = row_map; n.w = Y.final_norm; n.out = B->x;
        QB_TRY(qb_launch_layer_norm(ctx, n));
    }
    return qb_dense_gemm(ctx, Y.head, B->x, rows, dst, 1);
}

const QbArch ARCH_LAYERED = {"layered", 1024, layered_batch_alloc, layered_batch_free, layered_forward, layered_head, layered_model_free};

int layered_create(qb_ctx *ctx, const std::string &config, bool f32, Source &src, qb_model **out) {
    auto Y = std::make_unique<QbLayered>();
    QB_TRY(parse_spec(config, Y->spec));
    Y->f32 = f32;
    Y->runs = list_runs(Y->spec);
    Y->layers.resize(Y->spec.layers.size());
    QB_CUDA(cudaSetDevice(ctx->device));
    qb_model *m = new qb_model();
    m->arch = &ARCH_LAYERED;
    m->cfg = qb_model_config{};
    m->cfg.n_layers = (uint32_t)Y->spec.layers.size();
    m->cfg.n_embd = Y->spec.width;
    m->cfg.vocab_size = Y->spec.vocab;
    m->cfg.rms_eps = (float)Y->spec.eps;
    m->layered = Y.release();
    const int st = build_model(ctx, m, src);
    if (st != QB_OK) { qb_model_destroy(ctx, m); return st; }
    *out = m;
    return QB_OK;
}

}  // namespace

int qb_layered_load(qb_ctx *ctx, const char *dir, const std::string &config, bool f32, qb_model **out) {
    qbst::File file;
    QB_TRY(file.open((std::string(dir) + "/model.safetensors").c_str()));
    Source src;
    src.file = &file;
    return layered_create(ctx, config, f32, src, out);
}

extern "C" int qb_model_create_layered_synth(qb_ctx *ctx, const char *config_json, uint64_t seed, int f32, qb_model **out) {
    QB_REQUIRE(ctx && config_json && out, "qb_model_create_layered_synth: null argument");
    Source src;
    src.seed = seed;
    return layered_create(ctx, config_json, f32 != 0, src, out);
}

extern "C" int qb_debug_layer_trace(qb_ctx *ctx, qb_batch *b, int on) {
    QB_REQUIRE(ctx && b && b->layered, "qb_debug_layer_trace: a layered model's batch is needed");
    QB_CUDA(cudaStreamSynchronize(ctx->stream));
    if (b->layered->trace) cudaFree(b->layered->trace);
    b->layered->trace = nullptr;
    if (on) QB_CUDA(cudaMalloc(&b->layered->trace, b->m->layered->runs.size() * (size_t)b->rows_cap * b->m->cfg.n_embd * sizeof(float)));
    return QB_OK;
}
extern "C" int qb_debug_layer_trace_read(qb_ctx *ctx, qb_batch *b, float *host_out, uint32_t max_rows, uint32_t *runs_out, uint32_t *rows_out) {
    QB_REQUIRE(ctx && b && b->layered && b->layered->trace && runs_out && rows_out, "qb_debug_layer_trace_read: the trace is not on");
    const uint32_t D = b->m->cfg.n_embd, n = (uint32_t)b->m->layered->runs.size(), rows = std::min(max_rows, b->layered->trace_rows);
    *runs_out = n;
    *rows_out = rows;
    if (!host_out) return QB_OK;
    for (uint32_t r = 0; r < n; ++r)
        QB_CUDA(cudaMemcpyAsync(host_out + (size_t)r * rows * D, b->layered->trace + (size_t)r * b->rows_cap * D, (size_t)rows * D * sizeof(float),
                                cudaMemcpyDeviceToHost, ctx->stream));
    return qb_synchronize(ctx);
}
