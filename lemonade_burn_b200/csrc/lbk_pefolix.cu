// The Pefolix family of the model runtime: a decoder with layer norms before and after each sublayer, attention
// under a sliding window with kept first tokens and a distance bias (no rotation), and per layer either a gated
// feed-forward, a mixture of experts with a shared expert, or none. config.json lists the layers one by one; every
// size and constant comes from there or from a tensor's shape, so layers may differ from one another.
//
//   x = embed[token]
//   x += norm1b(W_o attention(norm1(x)));  x += norm2b(ff(norm2(x)))        per layer
//   logits = head final.norm(x)
//
// The residual, norms, scores, probabilities and routing are f32; activations between them are the compute type
// (bf16, or f32 for LBK_COMPUTE_F32). Launches of a layer of a decode step in bf16: [norms + q/k/v, k and v stored
// into the cache by the projection], attention (+ merge of its slices), o, [norms + gate/up + gelu product], down;
// with experts [norms + shared up + router + gate logit], chosen experts' up, all downs. A prompt pass runs the
// same calls on its rows. The cache is [seq][kv_heads][capacity][head] per layer, head sizes padded to 16.
#include "lbk_dense.cuh"
#include "lbk_runtime.cuh"

namespace lbk {

namespace {

struct PefolixLayer {
    // mixer
    size_t heads = 0, kv_heads = 0, dim = 0, vdim = 0, dimp = 0, vdimp = 0;
    float scale = 1.0f;
    AttnMask mask;
    DenseWeight qkv, o;
    float *norm1 = nullptr, *norm1b = nullptr, *norm2 = nullptr, *norm2b = nullptr;
    // feed-forward
    enum Kind { None, Dense, Moe } kind = None;
    size_t ff = 0;                  // dense, or one expert's
    DenseWeight gate_up, down;      // dense: [gate; up] stacked, down
    size_t experts = 0, top = 0, sff = 0;
    DenseWeight in;                 // [shared up; router; shared gate]: everything that reads the layer's input directly
    DenseWeight eup, edown, sdown;  // experts stacked
};

struct PefolixCache;

struct PefolixModel : Model {
    std::vector<PefolixLayer> layers;
    size_t width = 0;
    float eps = 0.0f;
    uint16_t *embed = nullptr;  // bf16 [vocab][width]
    DenseWeight head;           // bf16 [vocab][width], rows back to back
    float *final_norm = nullptr;
    size_t elem() const { return compute == LBK_COMPUTE_F32 ? 4 : 2; }
    int make_cache(size_t batch, size_t capacity, std::unique_ptr<Cache> &out) override;
    int make_prefill_buffers(Cache *c, size_t rows) override;
    int enqueue_step(Cache *c, cudaStream_t st) override;
    int enqueue_rows(Cache *c, size_t seq, size_t n, cudaStream_t st) override;
    int enqueue_head(const float *rows, size_t n, float *logits, cudaStream_t st) override;
    struct Work;
    int make_work(std::vector<void *> &owner, Work &w, size_t rows, size_t decode_b, size_t cap);
    int enqueue_tokens(PefolixCache *c, Work &w, const int32_t *tokens, size_t m, int seq, float *final_rows, cudaStream_t st);
};

// Buffers of one pass over `rows` tokens, sized for the largest layer. Rows of the compute type have a pitch of a
// multiple of 64 values; what lies past a row's end is zero or a number another layer left there, and meets the
// zero columns of the weights.
struct PefolixModel::Work {
    float *x = nullptr, *x2 = nullptr, *y = nullptr;
    void *n = nullptr, *q = nullptr, *attn = nullptr, *h = nullptr;
    float *z = nullptr, *ys = nullptr;
    void *hs = nullptr, *xs = nullptr, *eh = nullptr, *eo = nullptr;
    int *route = nullptr, *act = nullptr;
    float *scratch = nullptr;
};

struct PefolixCache : Cache {
    std::vector<void *> k, v;   // per layer [b][kv_heads][cap][dimp], [b][kv_heads][cap][vdimp]
    PefolixModel::Work step_work, rows_work;
    float *final_rows = nullptr;
};

int PefolixModel::make_work(std::vector<void *> &owner, Work &w, size_t rows, size_t decode_b, size_t cap) {
    const size_t es = elem();
    const bool few = rows <= LBK_GEMV_MAX_M && compute == LBK_COMPUTE_BF16;  // the few-token expert kernels take any pass of this size
    size_t q = 0, at = 0, h = 0, z = 0, hs = 0, xs = 0, eh = 0, eo = 0, route = 0, act = 0, scratch = 0;
    for (const PefolixLayer &l : layers) {
        q = std::max(q, l.heads * l.dimp);
        at = std::max(at, dense_pitch(l.heads * l.vdim));
        if (l.kind == PefolixLayer::Dense) h = std::max(h, dense_pitch(l.ff));
        if (l.kind == PefolixLayer::Moe) {
            z = std::max(z, l.experts + 1);
            hs = std::max(hs, dense_pitch(l.sff));
            // a pass of up to LBK_GEMV_MAX_M rows in a larger buffer still takes the few-token kernels
            const size_t few_rows = std::min<size_t>(rows, LBK_GEMV_MAX_M);
            eh = std::max(eh, rows * l.top * dense_pitch(l.ff));
            act = std::max(act, moe_few_act_ints(few_rows, l.experts, l.top));
            if (!few) {
                xs = std::max(xs, rows * l.top * dense_pitch(width));
                eo = std::max(eo, rows * l.top * dense_pitch(width));
                route = std::max(route, moe_route_ints(rows, l.experts, l.top));
            }
        }
        if (decode_b) scratch = std::max(scratch, attn_window_scratch(decode_b, l.heads, l.vdimp, attn_window_splits(cap, l.mask)));
    }
    struct { void **p; size_t bytes; } bufs[] = {
        {reinterpret_cast<void **>(&w.x), rows * width * 4}, {reinterpret_cast<void **>(&w.x2), rows * width * 4}, {reinterpret_cast<void **>(&w.y), rows * width * 4},
        {&w.n, rows * dense_pitch(width) * es}, {&w.q, rows * q * es}, {&w.attn, rows * at * es}, {&w.h, rows * h * es},
        {reinterpret_cast<void **>(&w.z), rows * z * 4}, {reinterpret_cast<void **>(&w.ys), z ? rows * width * 4 : 0}, {&w.hs, rows * hs * es},
        {&w.xs, compute == LBK_COMPUTE_BF16 ? xs * es : 0}, {&w.eh, eh * es}, {&w.eo, eo * es}, {reinterpret_cast<void **>(&w.route), route * 4},
        {reinterpret_cast<void **>(&w.act), act * 4}, {reinterpret_cast<void **>(&w.scratch), scratch * 4}};
    for (auto &b : bufs) {
        LBK_TRY(dev_alloc(owner, b.bytes, b.p));
        LBK_CUDA(cudaMemset(*b.p, 0, b.bytes ? b.bytes : 16));
    }
    return LBK_OK;
}

int PefolixModel::make_cache(size_t batch, size_t capacity, std::unique_ptr<Cache> &out) {
    PefolixCache *c = new PefolixCache();
    out.reset(c);
    if (capacity == 0) capacity = 4096;  // positions have no limit of their own
    if (capacity > (1u << 30)) return fail(LBK_ERR_UNSUPPORTED, "a cache of %zu positions", capacity);
    c->cap = capacity;
    for (const PefolixLayer &l : layers) {
        void *k = nullptr, *v = nullptr;
        const size_t rows = batch * l.kv_heads * capacity;
        LBK_TRY(dev_alloc(c->device_allocs, rows * l.dimp * elem(), &k));
        LBK_TRY(dev_alloc(c->device_allocs, rows * l.vdimp * elem(), &v));
        LBK_CUDA(cudaMemset(k, 0, rows * l.dimp * elem()));  // the padding of the head sizes stays zero
        LBK_CUDA(cudaMemset(v, 0, rows * l.vdimp * elem()));
        c->k.push_back(k);
        c->v.push_back(v);
    }
    LBK_TRY(make_work(c->device_allocs, c->step_work, batch, batch, capacity));
    LBK_TRY(dev_alloc(c->device_allocs, batch * width * 4, reinterpret_cast<void **>(&c->final_rows)));
    return LBK_OK;
}

int PefolixModel::make_prefill_buffers(Cache *cache, size_t rows) {
    PefolixCache *c = static_cast<PefolixCache *>(cache);
    return make_work(c->pf_allocs, c->rows_work, rows, 0, c->cap);
}

// `m` tokens through all layers: consecutive positions of sequence `seq`, or (seq < 0) one token of each sequence.
int PefolixModel::enqueue_tokens(PefolixCache *c, Work &w, const int32_t *tokens, size_t m, int seq, float *final_rows, cudaStream_t st) {
    const bool f32 = compute == LBK_COMPUTE_F32;
    const bool few = m <= LBK_GEMV_MAX_M && !f32;
    const bool fuse = !f32 && dense_pre_supported(m, width);  // the norms run inside the projection behind them
    const long npitch = static_cast<long>(dense_pitch(width));
    const int *pos = c->pos + (seq >= 0 ? seq : 0);
    LBK_TRY(lbk_embed_bf16(reinterpret_cast<lbk_ctx *>(ctx), embed, tokens, m, width, w.x, st));
    float *x = w.x, *x2 = w.x2;
    // what the sublayers so far still owe the residual: their output rows and the norm in front of the sum
    const float *y = nullptr, *w_post = nullptr;
    MoeOut moe;
    bool have_moe = false;

    auto norm_rows = [&](const float *w_next, void *out_e, float *out_f) -> int {
        NormCall n;
        n.compute = compute;
        n.x = x;
        n.y = have_moe ? nullptr : y;
        n.moe = have_moe ? &moe : nullptr;
        n.w_post = w_post;
        n.w = w_next;
        n.rows = m;
        n.n = width;
        n.eps = eps;
        n.out_e = out_e;
        n.lde = npitch;
        n.out_f = out_f;
        return launch_sandwich_norm(ctx, n, st);
    };
    // the projection `d` of the normed residual; `keep`: the normed rows are wanted in w.n as well
    auto project = [&](DenseCall &d, const float *w_next, bool keep) -> int {
        d.compute = compute;
        d.m = m;
        d.ldx = npitch;
        if (fuse && !have_moe) {
            d.pre.mode = y ? kPreAddNorm : kPreNorm;
            d.pre.x = x;
            d.pre.y = y;
            d.pre.w_post = w_post;
            d.pre.w = w_next;
            d.pre.xout = x2;
            d.pre.nout = keep ? w.n : nullptr;
            d.pre.ldn = npitch;
            d.pre.eps = eps;
            LBK_TRY(launch_dense(ctx, d, st));
            if (y) std::swap(x, x2);
        } else {
            LBK_TRY(norm_rows(w_next, w.n, nullptr));
            d.x = w.n;
            LBK_TRY(launch_dense(ctx, d, st));
        }
        y = nullptr;
        have_moe = false;
        return LBK_OK;
    };
    auto rows_f32 = [&](const void *in, const DenseWeight &wt, float *out) -> int {
        DenseCall d;
        d.compute = compute;
        d.m = m;
        d.x = in;
        d.ldx = static_cast<long>(wt.pitch);
        d.w = wt;
        d.out_rows = wt.rows;
        d.epi.kind = kEpiF32;
        d.epi.out = out;
        d.epi.ld = static_cast<long>(wt.rows);
        return launch_dense(ctx, d, st);
    };

    for (size_t li = 0; li < layers.size(); ++li) {
        const PefolixLayer &l = layers[li];
        {
            DenseCall d;
            d.w = l.qkv;
            d.out_rows = l.qkv.rows;
            d.epi.kind = kEpiQkv;
            d.epi.out = w.q;
            d.epi.ld = static_cast<long>(l.heads * l.dimp);
            d.epi.q_rows = static_cast<int>(l.heads * l.dim);
            d.epi.k_rows = static_cast<int>(l.kv_heads * l.dim);
            d.epi.dim = static_cast<int>(l.dim);
            d.epi.dimp = static_cast<int>(l.dimp);
            d.epi.vdim = static_cast<int>(l.vdim);
            d.epi.vdimp = static_cast<int>(l.vdimp);
            d.epi.kv_heads = static_cast<int>(l.kv_heads);
            d.epi.cap = static_cast<int>(c->cap);
            d.epi.kc = c->k[li];
            d.epi.vc = c->v[li];
            d.epi.pos = pos;
            d.epi.rows_of_seq = seq;
            d.epi.err_word = ctx->err_word;
            LBK_TRY(project(d, l.norm1, false));
        }
        {
            AttnCall a;
            a.compute = compute;
            a.q = w.q;
            a.kc = c->k[li];
            a.vc = c->v[li];
            a.pos = pos;
            a.n = m;
            a.rows_of_seq = seq;
            a.heads = l.heads;
            a.kv_heads = l.kv_heads;
            a.dim = l.dim;
            a.dimp = l.dimp;
            a.vdim = l.vdim;
            a.vdimp = l.vdimp;
            a.cap = c->cap;
            a.scale = l.scale;
            a.mask = l.mask;
            a.scratch = w.scratch;
            a.out = w.attn;
            a.ldo = static_cast<long>(l.o.pitch);
            LBK_TRY(launch_attn_window(ctx, a, st));
        }
        LBK_TRY(rows_f32(w.attn, l.o, w.y));
        y = w.y;
        w_post = l.norm1b;
        if (l.kind == PefolixLayer::Dense) {
            DenseCall d;
            d.w = l.gate_up;
            d.gated = true;
            d.up_row = d.out_rows = l.ff;
            d.epi.kind = kEpiElem;
            d.epi.out = w.h;
            d.epi.ld = static_cast<long>(l.down.pitch);
            LBK_TRY(project(d, l.norm2, false));
            LBK_TRY(rows_f32(w.h, l.down, w.y));
            y = w.y;
            w_post = l.norm2b;
        } else if (l.kind == PefolixLayer::Moe) {
            const long ldz = static_cast<long>(l.experts + 1);
            DenseCall d;
            d.w = l.in;
            d.out_rows = l.in.rows;
            d.epi.kind = kEpiElem;
            d.epi.act = kActRelu2;
            d.epi.out = w.hs;
            d.epi.ld = static_cast<long>(dense_pitch(l.sff));
            d.epi.f32_from = static_cast<int>(l.sff);
            d.epi.out2 = w.z;
            d.epi.ld2 = ldz;
            LBK_TRY(project(d, l.norm2, true));
            w_post = l.norm2b;
            if (few) {
                MoeFewCall f;
                f.n = static_cast<const uint16_t *>(w.n);
                f.ldn = npitch;
                f.m = m;
                f.z = w.z;
                f.ldz = ldz;
                f.experts = static_cast<int>(l.experts);
                f.top = static_cast<int>(l.top);
                f.up = l.eup;
                f.down = l.edown;
                f.ff = l.ff;
                f.width = width;
                f.h = static_cast<uint16_t *>(w.eh);
                f.hs = l.sff ? static_cast<const uint16_t *>(w.hs) : nullptr;
                f.shared_down = l.sdown;
                f.act = w.act;
                f.y = w.y;
                LBK_TRY(launch_moe_few(ctx, f, st));
                y = w.y;
            } else {
                MoeRoute r;
                moe_route_carve(r, w.route, m, l.experts, l.top);
                LBK_TRY(launch_moe_route(ctx, w.z, ldz, m, l.experts, l.top, r, f32 ? nullptr : w.n, npitch, f32 ? nullptr : w.xs, st));
                DenseCall up;
                up.compute = compute;
                up.x = f32 ? w.n : w.xs;
                up.gather = f32 ? r.token : nullptr;
                up.ldx = npitch;
                up.m = m * l.top;
                up.w = l.eup;
                up.out_rows = up.group_rows = l.ff;
                up.experts = static_cast<int>(l.experts);
                up.offs = r.offs;
                up.epi.kind = kEpiElem;
                up.epi.act = kActRelu2;
                up.epi.out = w.eh;
                up.epi.ld = static_cast<long>(l.edown.pitch);
                LBK_TRY(launch_dense(ctx, up, st));
                DenseCall dn = up;
                dn.x = w.eh;
                dn.gather = nullptr;
                dn.ldx = static_cast<long>(l.edown.pitch);
                dn.w = l.edown;
                dn.out_rows = dn.group_rows = width;
                dn.epi.act = kActNone;
                dn.epi.out = w.eo;
                dn.epi.ld = npitch;
                LBK_TRY(launch_dense(ctx, dn, st));
                if (l.sff) LBK_TRY(rows_f32(w.hs, l.sdown, w.ys));
                moe = MoeOut{};
                if (f32) moe.rows32 = static_cast<const float *>(w.eo);
                else moe.rows16 = static_cast<const uint16_t *>(w.eo);
                moe.place = r.place;
                moe.weight = r.weight;
                moe.top = static_cast<int>(l.top);
                moe.shared = l.sff ? w.ys : nullptr;
                moe.gate = w.z + l.experts;
                moe.ldg = ldz;
                moe.ld = npitch;
                have_moe = true;
            }
        }
    }
    return norm_rows(final_norm, nullptr, final_rows);
}

int PefolixModel::enqueue_step(Cache *cache, cudaStream_t st) {
    PefolixCache *c = static_cast<PefolixCache *>(cache);
    LBK_TRY(enqueue_tokens(c, c->step_work, c->tokens, c->b, -1, c->final_rows, st));
    return enqueue_head(c->final_rows, c->b, c->logits, st);
}

int PefolixModel::enqueue_rows(Cache *cache, size_t seq, size_t n, cudaStream_t st) {
    PefolixCache *c = static_cast<PefolixCache *>(cache);
    return enqueue_tokens(c, c->rows_work, c->pf_tokens, n, static_cast<int>(seq), c->pf_n, st);
}

int PefolixModel::enqueue_head(const float *rows, size_t n, float *logits, cudaStream_t st) {
    if (compute == LBK_COMPUTE_BF16) return lbk_bf16_linear(reinterpret_cast<lbk_ctx *>(ctx), rows, n, head.w, head.rows, head.cols, logits, st);
    DenseCall d;
    d.compute = compute;
    d.x = rows;
    d.ldx = static_cast<long>(width);
    d.m = n;
    d.w = head;
    d.out_rows = head.rows;
    d.epi.kind = kEpiF32;
    d.epi.out = logits;
    d.epi.ld = static_cast<long>(head.rows);
    return launch_dense(ctx, d, st);
}

// ---- loading --------------------------------------------------------------------------------------
int load_pefolix(Ctx *ctx, const std::string &dir, const Json &cj, int compute, int, int world, std::unique_ptr<Model> &out) {
    if (world > 1) return fail(LBK_ERR_UNSUPPORTED, "the Pefolix family is not sharded over ranks");
    PefolixModel *m = new PefolixModel();
    out.reset(m);
    m->ctx = ctx;
    m->compute = compute;
    const Json *layers = cj.get("layers"), *norm = cj.get("norm"), *eps = norm ? norm->get("eps") : nullptr;
    if (!layers || layers->kind != Json::Arr || layers->arr.empty()) return fail(LBK_ERR_INVALID, "%s/config.json: \"layers\" is missing or empty", dir.c_str());
    if (!eps || eps->kind != Json::Num) return fail(LBK_ERR_INVALID, "%s/config.json: norm.eps is missing", dir.c_str());
    m->eps = static_cast<float>(eps->num);
    TensorFile tf;
    LBK_TRY(tf.open_file(dir + "/model.safetensors", ctx->own_stream));
    WeightLoader ld{ctx, m->device_allocs, tf};
    size_t vocab = 0, width = 0, v2 = 0, w2 = 0;
    LBK_TRY(ld.shape("embed", &vocab, &width));
    LBK_TRY(ld.shape("head", &v2, &w2));
    size_t cv = 0, cw = 0;
    if (!vocab || !width || v2 != vocab || w2 != width || (json_positive(cj.get("vocab"), &cv) && cv != vocab) || (json_positive(cj.get("width"), &cw) && cw != width))
        return fail(LBK_ERR_SHAPE, "%s: embed is [%zu, %zu], head [%zu, %zu]; config.json says vocab %zu, width %zu", tf.path.c_str(), vocab, width, v2, w2, cv, cw);
    m->width = width;
    uint16_t *hd = nullptr;
    LBK_TRY(ld.table("embed", vocab, width, &m->embed));
    LBK_TRY(ld.table("head", vocab, width, &hd));
    m->head = DenseWeight{hd, vocab, width, width};
    LBK_TRY(ld.vec("final.norm", width, &m->final_norm));
    size_t first_ff = 0;
    for (size_t i = 0; i < layers->arr.size(); ++i) {
        const Json &lj = layers->arr[i];
        const std::string p = "l" + std::to_string(i) + ".";
        const Json *type = lj.get("type"), *mx = lj.get("mixer"), *mlp = lj.get("mlp");
        if (!type || type->kind != Json::Str || type->str != "attention" || !mx || mx->kind != Json::Obj)
            return fail(LBK_ERR_UNSUPPORTED, "%s/config.json: layer %zu has no mixer this family knows (attention)", dir.c_str(), i);
        PefolixLayer l;
        const Json *scale = mx->get("scale");
        if (!json_positive(mx->get("heads"), &l.heads) || !json_positive(mx->get("kv_heads"), &l.kv_heads) || !json_positive(mx->get("dim"), &l.dim) ||
            !json_positive(mx->get("vdim"), &l.vdim) || l.heads % l.kv_heads || !scale || scale->kind != Json::Num)
            return fail(LBK_ERR_INVALID, "%s/config.json: layer %zu: heads, kv_heads, dim, vdim or scale is missing or inconsistent", dir.c_str(), i);
        if (l.dim > 512 || l.vdim > 512) return fail(LBK_ERR_UNSUPPORTED, "layer %zu: head sizes of at most 512", i);
        l.dimp = pad16(l.dim);
        l.vdimp = pad16(l.vdim);
        l.scale = static_cast<float>(scale->num);
        const Json *mask = mx->get("mask");
        if (mask && mask->kind == Json::Obj) {
            size_t v = 0;
            if (json_positive(mask->get("size"), &v)) l.mask.size = static_cast<int>(v);
            if (json_positive(mask->get("keep_first"), &v)) l.mask.keep_first = static_cast<int>(v);
        }
        LBK_TRY(ld.vec(p + "norm1", width, &l.norm1));
        LBK_TRY(ld.vec(p + "norm1b", width, &l.norm1b));
        LBK_TRY(ld.stack({p + "mix.q", p + "mix.k", p + "mix.v"}, {l.heads * l.dim, l.kv_heads * l.dim, l.kv_heads * l.vdim}, width, &l.qkv));
        LBK_TRY(ld.stack({p + "mix.o"}, {width}, l.heads * l.vdim, &l.o));
        if (mlp && mlp->kind == Json::Obj) {
            LBK_TRY(ld.vec(p + "norm2", width, &l.norm2));
            LBK_TRY(ld.vec(p + "norm2b", width, &l.norm2b));
            const Json *kind = mlp->get("kind");
            const std::string ks = kind && kind->kind == Json::Str ? kind->str : "";
            size_t cols = 0;
            if (ks == "dense") {
                l.kind = PefolixLayer::Dense;
                LBK_TRY(ld.shape(p + "mlp.up", &l.ff, &cols));
                LBK_TRY(ld.stack({p + "mlp.gate", p + "mlp.up"}, {l.ff, l.ff}, width, &l.gate_up));
                LBK_TRY(ld.stack({p + "mlp.down"}, {width}, l.ff, &l.down));
                if (!first_ff) first_ff = l.ff;
            } else if (ks == "moe") {
                l.kind = PefolixLayer::Moe;
                const Json *router = mlp->get("router"), *shared = mlp->get("shared");
                if (!router || !json_positive(router->get("experts"), &l.experts) || !json_positive(router->get("top"), &l.top) || l.top > l.experts)
                    return fail(LBK_ERR_INVALID, "%s/config.json: layer %zu: mlp.router", dir.c_str(), i);
                if (l.experts > 1024 || l.top > 32) return fail(LBK_ERR_UNSUPPORTED, "layer %zu: at most 1024 experts, 32 of them per token", i);
                LBK_TRY(ld.shape(p + "mlp.e0.up", &l.ff, &cols));
                std::vector<std::string> in, ups, downs;
                std::vector<size_t> in_rows;
                if (shared && shared->kind == Json::Obj) {
                    LBK_TRY(ld.shape(p + "mlp.shared.up", &l.sff, &cols));
                    in.push_back(p + "mlp.shared.up");
                    in_rows.push_back(l.sff);
                }
                in.push_back(p + "mlp.router");
                in_rows.push_back(l.experts);
                if (l.sff) {
                    in.push_back(p + "mlp.shared.sg");
                    in_rows.push_back(1);
                    LBK_TRY(ld.stack({p + "mlp.shared.down"}, {width}, l.sff, &l.sdown));
                }
                LBK_TRY(ld.stack(in, in_rows, width, &l.in));
                for (size_t e = 0; e < l.experts; ++e) {
                    const std::string ep = p + "mlp.e" + std::to_string(e);
                    ups.push_back(ep + ".up");
                    downs.push_back(ep + ".down");
                }
                LBK_TRY(ld.stack(ups, std::vector<size_t>(l.experts, l.ff), width, &l.eup));
                LBK_TRY(ld.stack(downs, std::vector<size_t>(l.experts, width), l.ff, &l.edown));
                if (!first_ff) first_ff = l.ff;
            } else {
                return fail(LBK_ERR_UNSUPPORTED, "%s/config.json: layer %zu: unknown feed-forward \"%s\"", dir.c_str(), i, ks.c_str());
            }
        }
        m->layers.push_back(l);
    }
    LBK_CUDA(cudaStreamSynchronize(ctx->own_stream));  // the staging buffers go away now
    lbk_model_config &cfg = m->cfg;
    cfg.hidden_size = width;
    cfg.intermediate_size = first_ff;
    cfg.num_attention_heads = m->layers[0].heads;
    cfg.num_key_value_heads = m->layers[0].kv_heads;
    cfg.num_hidden_layers = m->layers.size();
    cfg.vocab_size = vocab;
    cfg.rms_norm_eps = m->eps;
    m->stats.bytes_read = tf.sg.bytes_read;
    m->stats.bytes_to_device = tf.sg.bytes_to_device;
    return LBK_OK;
}

const FamilyRegistrar kPefolix("Pefolix", load_pefolix);

}  // namespace

}  // namespace lbk
