// The BitNet b1.58 family of the model runtime: what lb-model's `BitNet::{load, new_cache, forward}`
// (crates/lb-model/src/model.rs:149-232, 234-236, 305-374) do, as launches of this library's kernels.
//
// Checkpoint: `config.json` + `model.lbt.safetensors` exactly as lb-convert writes them
// (crates/lb-convert/src/lib.rs:14-26: metadata format "lemonade-burn-ternary"; per linear
// `<name>.qweight` U8 [rows, padded(cols)/4] and `<name>.wscale` F32 [1]; norm gains F32; the tied
// embedding / LM head BF16). The packed weights go to the GPU as they are.
//
// Differences from the reference, all deliberate: the KV cache is bf16 with a fixed capacity
// (the reference grows an f32 cache, model.rs:245); several independent sequences can advance
// together (lbk_model_decode), which the reference cannot do. A prompt pass sends up to 4096 rows at a
// time through the projections (the tcgen05 GEMM above 16 rows) with causal attention over the cache, as
// the reference's forward does with m > 1.
#include "lbk_runtime.cuh"

namespace lbk {

namespace {

struct BitNetModel : Model {
    size_t head_dim = 0;
    struct Layer {
        lbk_weight *q = nullptr, *k = nullptr, *v = nullptr, *o = nullptr, *gate = nullptr, *up = nullptr, *down = nullptr;
        float *input_norm = nullptr, *post_attn_norm = nullptr, *attn_sub_norm = nullptr, *ffn_sub_norm = nullptr;
    };
    std::vector<Layer> layers;
    float *final_norm = nullptr;
    float *cos = nullptr, *sin = nullptr;
    uint16_t *embed = nullptr;  // bf16 [vocab][hidden], also the LM head (tied)
    std::vector<lbk_weight *> weights;
    ~BitNetModel() override {
        for (lbk_weight *w : weights) lbk_weight_free(w);
    }
    int make_cache(size_t batch, size_t capacity, std::unique_ptr<Cache> &out) override;
    int make_prefill_buffers(Cache *c, size_t rows) override;
    int enqueue_step(Cache *c, cudaStream_t st) override;
    int enqueue_rows(Cache *c, size_t seq, size_t n, cudaStream_t st) override;
    int enqueue_head(const float *rows, size_t n, float *logits, cudaStream_t st) override {
        return lbk_bf16_linear(reinterpret_cast<lbk_ctx *>(ctx), rows, n, embed, cfg.vocab_size, cfg.hidden_size, logits, st);
    }
};

struct BitNetCache : Cache {
    size_t splits = 1;
    uint16_t *k = nullptr, *v = nullptr;  // [layers][b][kv_heads][cap][head_dim]
    int32_t *counters = nullptr;
    float *x = nullptr, *x2 = nullptr, *n = nullptr, *q = nullptr, *kk = nullptr, *vv = nullptr, *attn = nullptr, *o = nullptr, *g = nullptr,
          *u = nullptr, *d = nullptr, *act = nullptr, *scratch = nullptr;
    int8_t *q8 = nullptr;  // quantised input rows of the next projection (batches of 9 and more)
    float *qscale = nullptr;
    int32_t *qsum = nullptr;
    float *pf_x = nullptr, *pf_q = nullptr, *pf_k = nullptr, *pf_v = nullptr, *pf_attn = nullptr, *pf_o = nullptr, *pf_g = nullptr,
          *pf_u = nullptr, *pf_act = nullptr, *pf_d = nullptr;
    int8_t *pf_q8 = nullptr;   // quantised input rows of the next projection (lbk_norm_quant)
    float *pf_qscale = nullptr;
    int32_t *pf_qsum = nullptr;
};

// model.rs:213-230: inv_freq in f32, angle = pos as f32 * inv_freq (f32), sin/cos evaluated in f64,
// stored as f32, the 64 values repeated for both halves of the head.
void rope_tables(const lbk_model_config &c, size_t hd, std::vector<float> &cs, std::vector<float> &sn) {
    const size_t half = hd / 2, np = c.max_position_embeddings;
    cs.resize(np * hd);
    sn.resize(np * hd);
    std::vector<float> inv(half);
    for (size_t i = 0; i < half; ++i) inv[i] = static_cast<float>(1.0 / std::pow(static_cast<double>(c.rope_theta), (2.0 * i) / hd));
    for (size_t p = 0; p < np; ++p)
        for (size_t i = 0; i < half; ++i) {
            const float ang = static_cast<float>(p) * inv[i];
            const float cv = static_cast<float>(std::cos(static_cast<double>(ang))), sv = static_cast<float>(std::sin(static_cast<double>(ang)));
            cs[p * hd + i] = cs[p * hd + half + i] = cv;
            sn[p * hd + i] = sn[p * hd + half + i] = sv;
        }
}

}  // namespace

// One decode step for cache->b sequences: the C++ twin of the Python mirror's BitNet.forward.
int BitNetModel::enqueue_step(Cache *cache, cudaStream_t st) {
    BitNetModel *m = this;
    BitNetCache *c = static_cast<BitNetCache *>(cache);
    lbk_ctx *h = reinterpret_cast<lbk_ctx *>(m->ctx);
    const lbk_model_config &cfg = m->cfg;
    const size_t b = c->b, H = cfg.hidden_size, I = cfg.intermediate_size, nh = cfg.num_attention_heads, kvh = cfg.num_key_value_heads,
                 hd = m->head_dim, L = cfg.num_hidden_layers;
    const float eps = cfg.rms_norm_eps;
    const bool pre_h = lbk_ternary_linear_pre_supported(b, H), pre_a = lbk_ternary_linear_pre_supported(b, nh * hd),
               pre_i = lbk_ternary_linear_pre_supported(b, I);
    const bool fused_norms = H % 4 == 0 && H <= 8192 && I % 4 == 0 && I <= 8192;
    const bool attn_fused = lbk_attn_decode_fused_supported(nh, kvh, hd, c->splits) != 0;
    const size_t layer_kv = b * kvh * c->cap * hd;
    float *x = c->x, *x2 = c->x2;
    auto add_norm = [&](float *xin, const float *y, const float *w) -> int {  // xin += y; n = rms_norm(xin) * w
        if (fused_norms) return lbk_add_rms_norm(h, xin, y, w, b, H, eps, c->n, st);
        LBK_TRY(lbk_add_inplace(h, xin, y, b * H, st));
        return lbk_rms_norm(h, xin, w, b, H, eps, c->n, st);
    };
    // From 9 sequences on every projection takes the quantise + GEMM path; the norm in front of it then
    // writes the quantised rows itself (lbk_norm_quant): no f32 copy, no quantise kernel. Same bits.
    const bool nq = b >= 9 && lbk_norm_quant_supported(H) && lbk_norm_quant_supported(I) && lbk_norm_quant_supported(nh * hd);
    auto norm_q = [&](int pre, float *xx, const float *yy, const float *w, size_t width) -> int {
        return lbk_norm_quant(h, pre, xx, yy, w, b, width, eps, c->q8, c->qscale, c->qsum, st);
    };
    auto proj_q = [&](const lbk_weight *const *ws, size_t nw, float *const *outs) -> int {
        return lbk_ternary_gemm_dev(h, ws, nw, c->q8, c->qscale, c->qsum, b, outs, nullptr, st);
    };
    LBK_TRY(lbk_embed_bf16(h, m->embed, c->tokens, b, H, x, st));
    bool have_d = false;  // c->d holds the previous layer's down projection, not yet added to x
    for (size_t li = 0; li < L; ++li) {
        const BitNetModel::Layer &l = m->layers[li];
        const lbk_weight *qkv[3] = {l.q, l.k, l.v};
        float *qkv_out[3] = {c->q, c->kk, c->vv};
        if (nq) {
            LBK_TRY(norm_q(have_d ? LBK_PRE_ADD_RMS : LBK_PRE_RMS, x, have_d ? c->d : nullptr, l.input_norm, H));
            LBK_TRY(proj_q(qkv, 3, qkv_out));
        } else if (!have_d) {
            if (pre_h) {
                LBK_TRY(lbk_ternary_linear_pre(h, LBK_PRE_RMS, x, nullptr, l.input_norm, eps, nullptr, b, qkv, 3, qkv_out, nullptr, st));
            } else {
                LBK_TRY(lbk_rms_norm(h, x, l.input_norm, b, H, eps, c->n, st));
                LBK_TRY(lbk_ternary_linear_n(h, c->n, b, qkv, 3, qkv_out, nullptr, st));
            }
        } else if (pre_h) {
            LBK_TRY(lbk_ternary_linear_pre(h, LBK_PRE_ADD_RMS, x, c->d, l.input_norm, eps, x2, b, qkv, 3, qkv_out, nullptr, st));
            std::swap(x, x2);
        } else {
            LBK_TRY(add_norm(x, c->d, l.input_norm));
            LBK_TRY(lbk_ternary_linear_n(h, c->n, b, qkv, 3, qkv_out, nullptr, st));
        }
        uint16_t *kc = c->k + li * layer_kv, *vc = c->v + li * layer_kv;
        if (attn_fused) {
            LBK_TRY(lbk_attn_decode_fused_seq(h, c->q, c->kk, c->vv, m->cos, m->sin, c->pos, b, nh, kvh, hd, c->cap, c->splits, kc, vc, c->scratch,
                                          c->counters, c->attn, st));
        } else {
            LBK_TRY(lbk_rope_kv_append_seq(h, c->q, c->kk, c->vv, m->cos, m->sin, c->pos, b, nh, kvh, hd, c->cap, kc, vc, st));
            LBK_TRY(lbk_attn_decode_seq(h, c->q, kc, vc, c->pos, b, nh, kvh, hd, c->cap, c->splits, c->scratch, c->attn, st));
        }
        const lbk_weight *ow[1] = {l.o};
        float *oo[1] = {c->o};
        if (nq) {
            const lbk_weight *gu[2] = {l.gate, l.up}, *dw[1] = {l.down};
            float *guo[2] = {c->g, c->u}, *dout[1] = {c->d};
            LBK_TRY(norm_q(LBK_PRE_RMS, c->attn, nullptr, l.attn_sub_norm, nh * hd));
            LBK_TRY(proj_q(ow, 1, oo));
            LBK_TRY(norm_q(LBK_PRE_ADD_RMS, x, c->o, l.post_attn_norm, H));
            LBK_TRY(proj_q(gu, 2, guo));
            LBK_TRY(norm_q(LBK_PRE_RELU2_MUL_RMS, c->g, c->u, l.ffn_sub_norm, I));
            LBK_TRY(proj_q(dw, 1, dout));
            have_d = true;
            continue;
        }
        if (pre_a) {
            LBK_TRY(lbk_ternary_linear_pre(h, LBK_PRE_RMS, c->attn, nullptr, l.attn_sub_norm, eps, nullptr, b, ow, 1, oo, nullptr, st));
        } else {
            LBK_TRY(lbk_rms_norm(h, c->attn, l.attn_sub_norm, b, nh * hd, eps, c->attn, st));
            LBK_TRY(lbk_ternary_linear_n(h, c->attn, b, ow, 1, oo, nullptr, st));
        }
        const lbk_weight *gu[2] = {l.gate, l.up};
        float *guo[2] = {c->g, c->u};
        if (pre_h) {
            LBK_TRY(lbk_ternary_linear_pre(h, LBK_PRE_ADD_RMS, x, c->o, l.post_attn_norm, eps, x2, b, gu, 2, guo, nullptr, st));
            std::swap(x, x2);
        } else {
            LBK_TRY(add_norm(x, c->o, l.post_attn_norm));
            LBK_TRY(lbk_ternary_linear_n(h, c->n, b, gu, 2, guo, nullptr, st));
        }
        const lbk_weight *dw[1] = {l.down};
        float *dout[1] = {c->d};
        if (pre_i) {
            LBK_TRY(lbk_ternary_linear_pre(h, LBK_PRE_RELU2_MUL_RMS, c->g, c->u, l.ffn_sub_norm, eps, nullptr, b, dw, 1, dout, nullptr, st));
        } else {
            if (fused_norms) {
                LBK_TRY(lbk_relu2_mul_rms_norm(h, c->g, c->u, l.ffn_sub_norm, b, I, eps, c->act, st));
            } else {
                LBK_TRY(lbk_relu2_mul(h, c->g, c->u, b * I, c->act, st));
                LBK_TRY(lbk_rms_norm(h, c->act, l.ffn_sub_norm, b, I, eps, c->act, st));
            }
            LBK_TRY(lbk_ternary_linear_n(h, c->act, b, dw, 1, dout, nullptr, st));
        }
        have_d = true;
    }
    if (have_d) LBK_TRY(add_norm(x, c->d, m->final_norm));
    else LBK_TRY(lbk_rms_norm(h, x, m->final_norm, b, H, eps, c->n, st));
    return enqueue_head(c->n, b, c->logits, st);
}

// About 150 KB per row at 2B4T shapes.
int BitNetModel::make_prefill_buffers(Cache *cache, size_t rows) {
    BitNetCache *c = static_cast<BitNetCache *>(cache);
    const size_t H = cfg.hidden_size, I = cfg.intermediate_size, nh = cfg.num_attention_heads, kvh = cfg.num_key_value_heads, hd = head_dim;
    struct { void **p; size_t bytes; } bufs[] = {
        {reinterpret_cast<void **>(&c->pf_x), rows * H * 4}, {reinterpret_cast<void **>(&c->pf_q), rows * nh * hd * 4},
        {reinterpret_cast<void **>(&c->pf_k), rows * kvh * hd * 4}, {reinterpret_cast<void **>(&c->pf_v), rows * kvh * hd * 4},
        {reinterpret_cast<void **>(&c->pf_attn), rows * nh * hd * 4}, {reinterpret_cast<void **>(&c->pf_o), rows * H * 4},
        {reinterpret_cast<void **>(&c->pf_g), rows * I * 4}, {reinterpret_cast<void **>(&c->pf_u), rows * I * 4},
        {reinterpret_cast<void **>(&c->pf_act), rows * I * 4}, {reinterpret_cast<void **>(&c->pf_d), rows * H * 4},
        {reinterpret_cast<void **>(&c->pf_q8), rows * (std::max(std::max(H, I), nh * hd) + 127) / 128 * 128},
        {reinterpret_cast<void **>(&c->pf_qscale), rows * 4}, {reinterpret_cast<void **>(&c->pf_qsum), rows * 4}};
    for (auto &bf : bufs) LBK_TRY(dev_alloc(c->pf_allocs, bf.bytes, bf.p));
    return LBK_OK;
}

// `n` consecutive tokens of sequence `seq` of the cache in one pass: the projections see n token rows (the
// tcgen05 GEMM above 16 rows), attention is causal over the cache (model.rs:305-374 with m = n).
int BitNetModel::enqueue_rows(Cache *cache, size_t seq, size_t n, cudaStream_t st) {
    BitNetModel *m = this;
    BitNetCache *c = static_cast<BitNetCache *>(cache);
    lbk_ctx *h = reinterpret_cast<lbk_ctx *>(ctx);
    const size_t H = cfg.hidden_size, I = cfg.intermediate_size, nh = cfg.num_attention_heads, kvh = cfg.num_key_value_heads, hd = head_dim,
                 L = cfg.num_hidden_layers;
    const float eps = cfg.rms_norm_eps;
    const bool fused_h = H % 4 == 0 && H <= 8192, fused_i = I % 4 == 0 && I <= 8192;
    auto add_norm = [&](float *x, const float *y, const float *w) -> int {  // x += y; pf_n = rms_norm(x) * w
        if (fused_h) return lbk_add_rms_norm(h, x, y, w, n, H, eps, c->pf_n, st);
        LBK_TRY(lbk_add_inplace(h, x, y, n * H, st));
        return lbk_rms_norm(h, x, w, n, H, eps, c->pf_n, st);
    };
    const size_t layer_kv = c->b * kvh * c->cap * hd;
    // From 9 rows on every projection takes the GEMM path, whose input is the quantised rows: the norm
    // in front of a projection then writes those directly (lbk_norm_quant) and the f32 copy of the
    // normalised rows, with the quantise kernel that would read it back, goes away. Same bits.
    const bool nq = n >= 9 && lbk_norm_quant_supported(H) && lbk_norm_quant_supported(I) && lbk_norm_quant_supported(nh * hd);
    auto norm_q = [&](int pre, float *x, const float *y, const float *w, size_t width) -> int {
        return lbk_norm_quant(h, pre, x, y, w, n, width, eps, c->pf_q8, c->pf_qscale, c->pf_qsum, st);
    };
    auto project = [&](const float *x_f32, const lbk_weight *const *ws, size_t nw, float *const *outs) -> int {
        if (nq) return lbk_ternary_gemm_dev(h, ws, nw, c->pf_q8, c->pf_qscale, c->pf_qsum, n, outs, nullptr, st);
        return lbk_ternary_linear_n(h, x_f32, n, ws, nw, outs, nullptr, st);
    };
    LBK_TRY(lbk_embed_bf16(h, m->embed, c->pf_tokens, n, H, c->pf_x, st));
    if (nq) LBK_TRY(norm_q(LBK_PRE_RMS, c->pf_x, nullptr, m->layers[0].input_norm, H));
    else LBK_TRY(lbk_rms_norm(h, c->pf_x, m->layers[0].input_norm, n, H, eps, c->pf_n, st));
    for (size_t li = 0; li < L; ++li) {
        const BitNetModel::Layer &l = m->layers[li];
        const lbk_weight *qkv[3] = {l.q, l.k, l.v};
        float *qkv_out[3] = {c->pf_q, c->pf_k, c->pf_v};
        LBK_TRY(project(c->pf_n, qkv, 3, qkv_out));
        uint16_t *kc = c->k + li * layer_kv, *vc = c->v + li * layer_kv;
        LBK_TRY(lbk_rope_kv_append_rows(h, c->pf_q, c->pf_k, c->pf_v, m->cos, m->sin, c->pos + seq, n, nh, kvh, hd, c->cap, seq, kc, vc, st));
        LBK_TRY(lbk_attn_prefill(h, c->pf_q, kc, vc, c->pos + seq, n, nh, kvh, hd, c->cap, seq, c->pf_attn, st));
        if (nq) LBK_TRY(norm_q(LBK_PRE_RMS, c->pf_attn, nullptr, l.attn_sub_norm, nh * hd));
        else LBK_TRY(lbk_rms_norm(h, c->pf_attn, l.attn_sub_norm, n, nh * hd, eps, c->pf_attn, st));
        const lbk_weight *ow[1] = {l.o};
        float *oo[1] = {c->pf_o};
        LBK_TRY(project(c->pf_attn, ow, 1, oo));
        if (nq) LBK_TRY(norm_q(LBK_PRE_ADD_RMS, c->pf_x, c->pf_o, l.post_attn_norm, H));
        else LBK_TRY(add_norm(c->pf_x, c->pf_o, l.post_attn_norm));
        const lbk_weight *gu[2] = {l.gate, l.up};
        float *guo[2] = {c->pf_g, c->pf_u};
        LBK_TRY(project(c->pf_n, gu, 2, guo));
        if (nq) {
            LBK_TRY(norm_q(LBK_PRE_RELU2_MUL_RMS, c->pf_g, c->pf_u, l.ffn_sub_norm, I));
        } else if (fused_i) {
            LBK_TRY(lbk_relu2_mul_rms_norm(h, c->pf_g, c->pf_u, l.ffn_sub_norm, n, I, eps, c->pf_act, st));
        } else {
            LBK_TRY(lbk_relu2_mul(h, c->pf_g, c->pf_u, n * I, c->pf_act, st));
            LBK_TRY(lbk_rms_norm(h, c->pf_act, l.ffn_sub_norm, n, I, eps, c->pf_act, st));
        }
        const lbk_weight *dw[1] = {l.down};
        float *dout[1] = {c->pf_d};
        LBK_TRY(project(c->pf_act, dw, 1, dout));
        if (nq && li + 1 < L) LBK_TRY(norm_q(LBK_PRE_ADD_RMS, c->pf_x, c->pf_d, m->layers[li + 1].input_norm, H));
        else LBK_TRY(add_norm(c->pf_x, c->pf_d, li + 1 < L ? m->layers[li + 1].input_norm : m->final_norm));
    }
    return LBK_OK;  // pf_n holds the final norm of every row
}

int BitNetModel::make_cache(size_t batch, size_t capacity, std::unique_ptr<Cache> &out) {
    if (world > 1)
        return fail(LBK_ERR_UNSUPPORTED, "this model holds shard %d of %d: its step needs the other ranks (drive it through the tensor-parallel layer calls)", rank, world);
    if (capacity == 0) capacity = cfg.max_position_embeddings;
    if (capacity > cfg.max_position_embeddings) return fail(LBK_ERR_INVALID, "capacity %zu exceeds max_position_embeddings %zu", capacity, cfg.max_position_embeddings);
    BitNetCache *c = new BitNetCache();
    out.reset(c);
    c->cap = capacity;
    const size_t H = cfg.hidden_size, I = cfg.intermediate_size, nh = cfg.num_attention_heads, kvh = cfg.num_key_value_heads, hd = head_dim;
    c->splits = std::min<size_t>((capacity + 31) / 32, 256);  // 32 positions per attention slice (the Python mirror's attention_splits)
    const size_t kv_elems = cfg.num_hidden_layers * batch * kvh * capacity * hd;
    LBK_TRY(dev_alloc(c->device_allocs, kv_elems * 2, reinterpret_cast<void **>(&c->k)));
    LBK_TRY(dev_alloc(c->device_allocs, kv_elems * 2, reinterpret_cast<void **>(&c->v)));
    LBK_CUDA(cudaMemset(c->k, 0, kv_elems * 2));
    LBK_CUDA(cudaMemset(c->v, 0, kv_elems * 2));
    struct { void **p; size_t bytes; } bufs[] = {
        {reinterpret_cast<void **>(&c->counters), batch * kvh * 4}, {reinterpret_cast<void **>(&c->x), batch * H * 4},
        {reinterpret_cast<void **>(&c->x2), batch * H * 4}, {reinterpret_cast<void **>(&c->n), batch * H * 4},
        {reinterpret_cast<void **>(&c->q), batch * nh * hd * 4}, {reinterpret_cast<void **>(&c->kk), batch * kvh * hd * 4},
        {reinterpret_cast<void **>(&c->vv), batch * kvh * hd * 4}, {reinterpret_cast<void **>(&c->attn), batch * nh * hd * 4},
        {reinterpret_cast<void **>(&c->o), batch * H * 4}, {reinterpret_cast<void **>(&c->g), batch * I * 4}, {reinterpret_cast<void **>(&c->u), batch * I * 4},
        {reinterpret_cast<void **>(&c->d), batch * H * 4}, {reinterpret_cast<void **>(&c->act), batch * I * 4},
        {reinterpret_cast<void **>(&c->q8), batch * ((std::max(std::max(H, I), nh * hd) + 127) / 128 * 128)},
        {reinterpret_cast<void **>(&c->qscale), batch * 4}, {reinterpret_cast<void **>(&c->qsum), batch * 4},
        {reinterpret_cast<void **>(&c->scratch), batch * nh * c->splits * (hd + 4) * 4}};
    for (auto &bf : bufs) {
        LBK_TRY(dev_alloc(c->device_allocs, bf.bytes, bf.p));
        LBK_CUDA(cudaMemset(*bf.p, 0, bf.bytes));
    }
    return LBK_OK;
}

// ---- loader ------------------------------------------------------------------------------------
// The reference maps the file and copies every tensor into a framework tensor, which doubles its
// resident memory while loading (crates/lb-model/src/model.rs:172-183, docs/BENCHMARKS.md:57-59).
// Here tensor bytes go file -> one of two pinned staging buffers (pread) -> device (one
// cudaMemcpyAsync / cudaMemcpy2DAsync per piece on the context's stream); a buffer is refilled while
// the other one's copy is in flight. The host never holds more than the two buffers, whatever the
// model's size. All packed weights live in ONE device arena (256-byte aligned slices, wrapped as
// weights without a copy).
//
// Tensor parallel (rank, world): q/k/v/gate/up keep their row range [rank*rows/world, ...), which is a
// contiguous byte range of the file (rows are contiguous in the lb-ternary layout, pack.rs:46-49);
// o/down keep a column range that is a multiple of 128 columns, i.e. bytes [rank*rb/world, ...) of
// every packed row, cut out by a strided copy from the staging buffer. Norm gains, the embedding
// (also the head; a rank uses vocabulary rows [rank*V/world, ...) of it) and the RoPE tables are
// whole on every rank.
namespace {

int load_bitnet(Ctx *ctx, const std::string &dir, const Json &cj, int compute, int rank, int world, std::unique_ptr<Model> &out) {
    if (compute != LBK_COMPUTE_BF16) return fail(LBK_ERR_UNSUPPORTED, "the BitNet family computes in its own precisions only (int8 dots, bf16 cache)");
    lbk_ctx *c = reinterpret_cast<lbk_ctx *>(ctx);
    const char *directory = dir.c_str();
    BitNetModel *m = new BitNetModel();
    out.reset(m);
    m->ctx = ctx;
    m->rank = rank;
    m->world = world;
    bool ok = true;
    lbk_model_config &cfg = m->cfg;
    cfg.hidden_size = json_size(cj.get("hidden_size"), ok);
    cfg.intermediate_size = json_size(cj.get("intermediate_size"), ok);
    cfg.num_attention_heads = json_size(cj.get("num_attention_heads"), ok);
    cfg.num_key_value_heads = json_size(cj.get("num_key_value_heads"), ok);
    cfg.num_hidden_layers = json_size(cj.get("num_hidden_layers"), ok);
    cfg.vocab_size = json_size(cj.get("vocab_size"), ok);
    cfg.max_position_embeddings = json_size(cj.get("max_position_embeddings"), ok);
    const Json *je = cj.get("rms_norm_eps"), *jt = cj.get("rope_theta");
    if (!je || je->kind != Json::Num || !jt || jt->kind != Json::Num) ok = false;
    if (!ok) return fail(LBK_ERR_INVALID, "%s/config.json: a required field is missing or not a number", directory);
    cfg.rms_norm_eps = static_cast<float>(je->num);
    cfg.rope_theta = static_cast<float>(jt->num);
    const Json *jb = cj.get("bos_token_id");
    cfg.bos_token_id = jb && jb->kind == Json::Num ? static_cast<int>(jb->num) : 0;
    // model.rs:151-153: only the relu2, tied-embedding family
    // (both fields are required members of the reference's Config, model.rs:22-36: a file without them does not load there either)
    const Json *ja = cj.get("hidden_act"), *jtie = cj.get("tie_word_embeddings");
    if (!ja || !jtie) return fail(LBK_ERR_INVALID, "%s/config.json: missing field %s", directory, !ja ? "hidden_act" : "tie_word_embeddings");
    if (!(ja->kind == Json::Str && ja->str == "relu2")) return fail(LBK_ERR_UNSUPPORTED, "unsupported config: hidden_act must be relu2");
    if (!(jtie->kind == Json::Bool && jtie->b)) return fail(LBK_ERR_UNSUPPORTED, "unsupported config: tie_word_embeddings must be true");
    if (!cfg.num_attention_heads || !cfg.num_key_value_heads || cfg.hidden_size % cfg.num_attention_heads ||
        cfg.num_attention_heads % cfg.num_key_value_heads || !cfg.num_hidden_layers || !cfg.max_position_embeddings)
        return fail(LBK_ERR_INVALID, "config.json: inconsistent head counts or sizes");
    m->head_dim = cfg.hidden_size / cfg.num_attention_heads;
    if (m->head_dim != 128) return fail(LBK_ERR_UNSUPPORTED, "the attention kernels are built for head_dim 128, this model has %zu", m->head_dim);
    const size_t H = cfg.hidden_size, I = cfg.intermediate_size, hd = m->head_dim, W = static_cast<size_t>(world);
    if (world > 1 && (cfg.num_key_value_heads % W || I % (128 * W) || (cfg.num_attention_heads * hd) % (128 * W) || cfg.vocab_size % W))
        return fail(LBK_ERR_UNSUPPORTED, "%d ranks do not divide this model: KV heads %zu, intermediate %zu and attention width %zu (in blocks of 128 columns), vocabulary %zu",
                    world, cfg.num_key_value_heads, I, cfg.num_attention_heads * hd, cfg.vocab_size);

    // ---- model.lbt.safetensors: u64 header length, JSON header, data -------------------------
    TensorFile tf;
    LBK_TRY(tf.open_file(dir + "/model.lbt.safetensors", ctx->own_stream));
    if (tf.format != "lemonade-burn-ternary")  // model.rs:158-161
        return fail(LBK_ERR_INVALID, "%s is not a lemonade-burn ternary file (format=%s)", tf.path.c_str(), tf.format.empty() ? "none" : tf.format.c_str());
    Stager &sg = tf.sg;
    // norm gains (model.rs:165: F32) share one small arena
    const size_t L = cfg.num_hidden_layers;
    float *norms = nullptr;
    LBK_TRY(dev_alloc(m->device_allocs, (L * (3 * H + I) + H) * 4, reinterpret_cast<void **>(&norms)));
    size_t norm_off = 0;
    auto load_vec = [&](const std::string &name, size_t elems, float **dst) -> int {
        const TensorEntry *e;
        LBK_TRY(tf.find(name, "F32", elems, 4, &e));
        *dst = norms + norm_off;
        norm_off += elems;
        return sg.copy_linear(e->begin, elems * 4, *dst, name.c_str());
    };
    // one arena for every packed matrix of this rank
    struct Lin { const char *name; size_t rows, cols; bool split_cols; };
    const Lin lins[7] = {{".self_attn.q_proj", cfg.num_attention_heads * hd, H, false}, {".self_attn.k_proj", cfg.num_key_value_heads * hd, H, false},
                         {".self_attn.v_proj", cfg.num_key_value_heads * hd, H, false}, {".self_attn.o_proj", H, cfg.num_attention_heads * hd, true},
                         {".mlp.gate_proj", I, H, false}, {".mlp.up_proj", I, H, false}, {".mlp.down_proj", H, I, true}};
    size_t arena_bytes = 0;
    for (const Lin &ln : lins) {
        const size_t rows = ln.split_cols ? ln.rows : ln.rows / W, cols = ln.split_cols ? ln.cols / W : ln.cols;
        arena_bytes += (rows * lbk_row_bytes(cols) + 255) / 256 * 256;
    }
    arena_bytes *= L;
    unsigned char *arena = nullptr;
    LBK_TRY(dev_alloc(m->device_allocs, arena_bytes, reinterpret_cast<void **>(&arena)));
    size_t arena_off = 0;
    m->layers.resize(L);
    for (size_t i = 0; i < L; ++i) {
        const std::string p = "model.layers." + std::to_string(i);
        BitNetModel::Layer &l = m->layers[i];
        LBK_TRY(load_vec(p + ".input_layernorm.weight", H, &l.input_norm));
        LBK_TRY(load_vec(p + ".post_attention_layernorm.weight", H, &l.post_attn_norm));
        LBK_TRY(load_vec(p + ".self_attn.attn_sub_norm.weight", H, &l.attn_sub_norm));
        LBK_TRY(load_vec(p + ".mlp.ffn_sub_norm.weight", I, &l.ffn_sub_norm));
        lbk_weight **dst[7] = {&l.q, &l.k, &l.v, &l.o, &l.gate, &l.up, &l.down};
        for (int k = 0; k < 7; ++k) {
            const Lin &ln = lins[k];
            const std::string name = p + ln.name;
            const TensorEntry *es, *ew;
            LBK_TRY(tf.find(name + ".wscale", "F32", 1, 4, &es));
            float scale = 0.0f;
            if (pread(sg.fd, &scale, 4, static_cast<off_t>(sg.data0 + es->begin)) != 4) return fail(LBK_ERR_INVALID, "cannot read %s.wscale", name.c_str());
            const size_t rb = lbk_row_bytes(ln.cols);
            LBK_TRY(tf.find(name + ".qweight", "U8", ln.rows * rb, 1, &ew));
            unsigned char *dev = arena + arena_off;
            size_t rows = ln.rows, cols = ln.cols;
            if (!ln.split_cols) {
                rows = ln.rows / W;
                LBK_TRY(sg.copy_linear(ew->begin + static_cast<size_t>(rank) * rows * rb, rows * rb, dev, name.c_str()));
            } else if (world == 1) {
                LBK_TRY(sg.copy_linear(ew->begin, rows * rb, dev, name.c_str()));
            } else {
                cols = ln.cols / W;
                const size_t width = rb / W;
                LBK_TRY(sg.copy_columns(ew->begin, rows, rb, static_cast<size_t>(rank) * width, width, dev, name.c_str()));
            }
            arena_off += (rows * lbk_row_bytes(cols) + 255) / 256 * 256;
            LBK_TRY(lbk_weight_wrap(c, rows, cols, dev, scale, dst[k]));
            m->weights.push_back(*dst[k]);
        }
    }
    LBK_TRY(load_vec("model.norm.weight", H, &m->final_norm));
    const TensorEntry *ee;
    LBK_TRY(tf.find("model.embed_tokens.weight", "BF16", cfg.vocab_size * H, 2, &ee));  // model.rs:204
    LBK_TRY(dev_alloc(m->device_allocs, cfg.vocab_size * H * 2, reinterpret_cast<void **>(&m->embed)));
    LBK_TRY(sg.copy_linear(ee->begin, cfg.vocab_size * H * 2, m->embed, "model.embed_tokens.weight"));
    std::vector<float> cs, sn;
    rope_tables(cfg, hd, cs, sn);
    LBK_TRY(dev_alloc(m->device_allocs, cs.size() * 4, reinterpret_cast<void **>(&m->cos)));
    LBK_TRY(dev_alloc(m->device_allocs, sn.size() * 4, reinterpret_cast<void **>(&m->sin)));
    LBK_CUDA(cudaMemcpyAsync(m->cos, cs.data(), cs.size() * 4, cudaMemcpyHostToDevice, ctx->own_stream));
    LBK_CUDA(cudaMemcpyAsync(m->sin, sn.data(), sn.size() * 4, cudaMemcpyHostToDevice, ctx->own_stream));
    LBK_CUDA(cudaStreamSynchronize(ctx->own_stream));  // also: `cs`, `sn` and the staging buffers go away now
    m->stats.bytes_read = sg.bytes_read;
    m->stats.bytes_to_device = sg.bytes_to_device;
    return LBK_OK;
}

const FamilyRegistrar kBitNet("", load_bitnet);

}  // namespace

}  // namespace lbk

using namespace lbk;

extern "C" {

const lbk_weight *lbk_model_linear(const lbk_model *mp, size_t layer, int which) {
    const BitNetModel *m = dynamic_cast<const BitNetModel *>(reinterpret_cast<const Model *>(mp));
    if (!m || layer >= m->layers.size()) return nullptr;
    const BitNetModel::Layer &l = m->layers[layer];
    switch (which) {
        case LBK_LIN_Q: return l.q;
        case LBK_LIN_K: return l.k;
        case LBK_LIN_V: return l.v;
        case LBK_LIN_O: return l.o;
        case LBK_LIN_GATE: return l.gate;
        case LBK_LIN_UP: return l.up;
        case LBK_LIN_DOWN: return l.down;
        default: return nullptr;
    }
}

const float *lbk_model_norm(const lbk_model *mp, size_t layer, int which) {
    const BitNetModel *m = dynamic_cast<const BitNetModel *>(reinterpret_cast<const Model *>(mp));
    if (!m) return nullptr;
    if (which == LBK_NORM_FINAL) return m->final_norm;
    if (layer >= m->layers.size()) return nullptr;
    const BitNetModel::Layer &l = m->layers[layer];
    switch (which) {
        case LBK_NORM_INPUT: return l.input_norm;
        case LBK_NORM_POST_ATTN: return l.post_attn_norm;
        case LBK_NORM_ATTN_SUB: return l.attn_sub_norm;
        case LBK_NORM_FFN_SUB: return l.ffn_sub_norm;
        default: return nullptr;
    }
}

const uint16_t *lbk_model_embedding(const lbk_model *mp) {
    const BitNetModel *m = dynamic_cast<const BitNetModel *>(reinterpret_cast<const Model *>(mp));
    return m ? m->embed : nullptr;
}
const float *lbk_model_rope_cos(const lbk_model *mp) {
    const BitNetModel *m = dynamic_cast<const BitNetModel *>(reinterpret_cast<const Model *>(mp));
    return m ? m->cos : nullptr;
}
const float *lbk_model_rope_sin(const lbk_model *mp) {
    const BitNetModel *m = dynamic_cast<const BitNetModel *>(reinterpret_cast<const Model *>(mp));
    return m ? m->sin : nullptr;
}

}  // extern "C"
