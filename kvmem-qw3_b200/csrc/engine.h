// Structures shared by the executor (engine.cu) and the model families it drives.
#pragma once

#include "page_pool.h"
#include "qb_internal.h"

#include <string>

struct QbLayered;
struct QbLayeredBatch;

struct RowSet {
    uint32_t seq0 = 0, ns = 0, R = 0;      // sequences [seq0, seq0+ns), R rows each
    const int32_t *seq_pos = nullptr;      // device [ns]: position of each sequence's first row
    uint32_t max_pos = 0;                  // host upper bound of any row position
    bool ingest = false;                   // rows of a prompt chunk (not of a decode / verify step)
    uint32_t rows() const { return ns * R; }
};

// A model family.  The executor owns positions, page tables, slots, sampling and the step records; a family allocates its
// caches and activations for a batch, runs rows through its layers and turns hidden rows into logits.
struct QbArch {
    const char *name;
    uint32_t chunk;                      // rows of a prompt chunk
    int (*batch_alloc)(qb_ctx *ctx, qb_batch *b, size_t slots);     // slots: K/V positions the paged caches hold
    void (*batch_free)(qb_batch *b);
    // Leaves the residual rows in b->hid[0 .. rows).  checkpoints: keep the recurrent state after every row (verify rows).
    int (*forward)(qb_ctx *ctx, qb_batch *b, const int32_t *tokens_dev, const RowSet &rs, bool checkpoints);
    // dst[rows][vocab] = logits of the rows just forwarded (row_map null) or of b->hid rows row_map[0 .. rows).
    int (*head)(qb_ctx *ctx, qb_batch *b, const int32_t *row_map, uint32_t rows, float *dst);
    void (*model_free)(qb_ctx *ctx, qb_model *m);
};
// Loader of a model folder: config.json names the architecture.  f32: every product and activation in 32 bits.
struct QbLoader {
    const char *architecture;
    int (*load)(qb_ctx *ctx, const char *dir, const std::string &config, bool f32, qb_model **out);
};
int qb_layered_load(qb_ctx *ctx, const char *dir, const std::string &config, bool f32, qb_model **out);

// Per-sequence recurrent state: [n_seqs][per_seq] floats, of which the first `head` matter at the end of a prompt chunk.
// A ping-pong pair (buf[1] set) holds the valid copy in buf[conv_par].
struct StateBlock {
    float *buf[2] = {nullptr, nullptr};
    size_t per_seq = 0, head = 0;
};

struct LayerW {
    bool recurrent = false;
    qb_weight *w_in = nullptr;       // attention: [q(+gate) ; k ; v]   DeltaNet: [qkv ; z ; alpha ; beta]
    qb_weight *w_out = nullptr;      // attn_output / ssm_out
    qb_weight *w_gate_up = nullptr;  // [gate ; up]
    qb_weight *w_down = nullptr;
    qb_weight w_kv;                  // view of the k and v rows of w_in (attention layers)
    float *conv_w = nullptr, *ssm_a = nullptr, *dt_bias = nullptr;
    // RMSNorm gains (attn_norm, ffn_norm / post_attention_norm, attn_q_norm, attn_k_norm, ssm_norm)
    const float *attn_norm = nullptr, *ffn_norm = nullptr, *q_norm = nullptr, *k_norm = nullptr, *ssm_norm = nullptr;
};

struct qb_model {
    qb_model_config cfg;
    const QbArch *arch = nullptr;    // the family: forward pass and per-batch buffers
    QbLayered *layered = nullptr;    // a layered model's description and weights (layered_model.cu)
    std::vector<LayerW> layers;      // n_layers (+ the MTP layer last)
    qb_weight *token_embd = nullptr, *output = nullptr, *eh_proj = nullptr;
    // MTP head: embedding table and LM head (nextn.embed_tokens / nextn.shared_head_head, else the target's)
    qb_weight *mtp_embd = nullptr, *mtp_head = nullptr;
    bool output_tied = false;        // no output.weight: the LM head is token_embd
    uint32_t tp_rank = 0, tp_world = 1;   // FFN weights are shard tp_rank of tp_world (tensor-parallel form), else whole
    float *ones = nullptr;           // every RMSNorm gain of the seeded model is 1.0
    const float *output_norm = nullptr, *enorm = nullptr, *hnorm = nullptr, *shared_head_norm = nullptr;
    std::vector<float *> owned_f32;  // fp32 tensors uploaded for this model
    float *inv_freq = nullptr;
    size_t weight_bytes = 0;
    uint32_t inner() const { return cfg.n_heads * cfg.head_dim; }
    uint32_t kvd() const { return cfg.n_kv_heads * cfg.head_dim; }
    uint32_t attn_in() const { return 2 * inner() + 2 * kvd(); }
    uint32_t qkv_dim() const { return (2 * cfg.ssm_num_k_heads + cfg.ssm_num_v_heads) * cfg.ssm_head_dim; }
    uint32_t vdim() const { return cfg.ssm_num_v_heads * cfg.ssm_head_dim; }
    uint32_t dn_in() const { return qkv_dim() + vdim() + 2 * cfg.ssm_num_v_heads; }
    bool is_attn(uint32_t i) const { return cfg.full_attention_interval && ((i + 1) % cfg.full_attention_interval) == 0; }
};

struct QBuf {   // quantised activation buffer for one K
    int8_t *q = nullptr; float *d = nullptr; uint32_t K = 0;
};

struct qb_batch {
    qb_model *m = nullptr;
    QbLayeredBatch *layered = nullptr;     // a layered model's caches and activations (layered_model.cu)
    std::vector<StateBlock> blocks;        // recurrent state of every kind: reset, swap, snapshot and prefix entries walk this list
    size_t slots = 0;                      // K/V positions the paged caches hold
    uint32_t n_seqs = 0, max_ctx = 0, k = 0, page_size = 0, pages_per_seq = 0, rows_cap = 0, chunk = 0, logit_rows = 0;
    bool attn_tc = false;                  // decode / verify attention on the tensor-memory kernel: decided once, from n_seqs * max_ctx
    uint32_t attn_split = 0;               // keys per attention split of this batch (absolute boundaries): decided once with attn_tc
    uint32_t n_active = 0;                 // the decode steps run sequences [0, n_active); the rest keep their state untouched
    std::vector<__half *> kc, vc;          // per layer (attention layers only), + MTP layer at index n_layers
    std::vector<float *> state, conv;      // per layer (recurrent layers only): [n_seqs][k+1][...]
    std::vector<float *> conv_alt;         // second conv-state buffer: a forward reads one and writes the other
    int conv_par = 0;                      // which of the two holds the valid conv state (the same for all sequences)
    int32_t *page_table = nullptr;         // [n_seqs][pages_per_seq]
    // pooled form (qb_batch_create_pooled): the caches hold pool->total() pages shared by all sequences; a sequence's
    // page-table row grows as its position grows and goes back to the pool at qb_seq_reset
    QbPagePool *pool = nullptr;
    std::vector<std::vector<int32_t>> seq_pages;   // host mirror of the page-table rows (pooled form)
    std::vector<int32_t> chunk_end_pos;            // position after the sequence's last qb_prefill_chunk, -1 once anything else moved it
    // device control block (all int32)
    int32_t *ctl = nullptr;
    int32_t *pos = nullptr, *sel = nullptr, *cur = nullptr, *drafts = nullptr, *zero_sel = nullptr;
    int32_t *tok_buf = nullptr, *seqpos_buf = nullptr, *prefix_pos = nullptr, *prefix_tok = nullptr;
    int32_t *out_rec = nullptr;            // [n_out (n_seqs) | tokens (n_seqs*(k+1)) | pos (n_seqs)]
    int32_t *map_prevh = nullptr, *map_prefix = nullptr, *map_chunk = nullptr, *map_last = nullptr;
    long long *stats = nullptr;            // [QB_STATS]: steps, drafted, accepted, emitted, rejecting steps, -, -, -, then steps by accepted length
    int32_t *out_rec_host = nullptr;       // pinned mirror of out_rec
    // activations
    float *hid = nullptr;                  // [rows_cap + n_seqs][H]; rows rows_cap+s hold prev hidden of seq s
    float *mtp_h = nullptr, *embd = nullptr, *act = nullptr, *parts = nullptr;
    float *logits = nullptr, *am_val = nullptr, *att_acc = nullptr, *att_ml = nullptr;
    int32_t *am_idx = nullptr;
    QBuf xq_h, xq_attn, xq_dn, xq_ffn, xq_cat;
    size_t parts_floats = 0;
    std::vector<int32_t> host_pos;         // upper bound of pos per sequence
    uint32_t last_logit_rows = 0;
    float *score_logits = nullptr;         // logits of chosen prompt rows (qb_prefill_logits) and the rows they come from
    int32_t *score_map = nullptr;
    int gemm_impl = 0;
    double *samp_u = nullptr;              // [2][logit_rows]: acceptance draws, then residual draws (sampling mode)
    uint32_t *seen = nullptr;              // [n_seqs][seen_words] bitmap of prompt + emitted tokens (token penalties), or null
    uint32_t seen_words = 0;
    float pen_presence = 0.0f, pen_repetition = 1.0f;
    qb_tp_group *tp = nullptr;             // tensor-parallel FFN group of the batch's model shard, or null
    float *normed = nullptr, *tp_y = nullptr;   // [rows_cap][H]: fp32 FFN input / all-reduced FFN output of the tensor-parallel form
    int32_t *tok_stage = nullptr;          // pinned staging of the prompt tokens being ingested
    int32_t *tok_all = nullptr;            // the same on the device: one copy per call, the chunks index into it
    cudaEvent_t tok_ev = nullptr;          // that copy has landed (the staging area may be rewritten)
    uint32_t tok_stage_cap = 0;
    double *first_draw_stage = nullptr;    // pinned: the first-token draw of a sampled request per sequence
    int32_t *limit = nullptr;              // [n_seqs] device: draft depth of the next step per sequence (<= k)
    int32_t *limit_host = nullptr;         // pinned staging of the same
    int32_t eos_token = -1;                // a draft equal to it ends the chain (-1: none)
    void *swap_tmp = nullptr;              // one sequence's largest per-layer state block (qb_seq_swap)
    size_t swap_bytes = 0;
    // sampled steps: pinned staging ring of the step's draws (a slot is reused when its copy of four steps ago has landed)
    static constexpr int SAMP_RING = 4;
    double *samp_stage = nullptr;
    cudaEvent_t samp_ev[SAMP_RING] = {};
    uint32_t samp_slot = 0;
    // position probe: keeps host_pos near the device's positions when nobody reads the step records (see probe_tick)
    int32_t *probe_host = nullptr;         // pinned [n_seqs]
    cudaEvent_t probe_ev = nullptr;
    bool probe_pending = false;
    int32_t probe_adv = 0;                 // positions enqueued since the probe's copy
    uint32_t steps_since_probe = 0;
};

int qb_upload_f32(qb_ctx *ctx, const std::vector<float> &v, float **out);
