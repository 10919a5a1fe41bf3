// The Dugulorn family of the model runtime: a decoder whose layers each have one of three mixers (latent attention,
// lightning attention, gated delta rule with a decay per channel) and a squared-relu feed-forward with biases or none.
// Sublayers read the residual itself; only their outputs are normed. config.json lists the layers one by one; every size
// and constant comes from there or from a tensor's shape, so layers may differ from one another.
//
//   x = norm(embed[token])
//   x += norm1(mixer(x));  x += norm2(ff(x))              per layer
//   logits = embed norm(x)
//
// norm: x / sqrt(mean(x^2) + eps) * (1 + w); the 1 is added when the weights are loaded. The residual, norms, angles,
// scores, probabilities, decays, step sizes and recurrent states are f32; activations between them are the compute type
// (bf16, or f32 for LBK_COMPUTE_F32). What a sequence holds: per latent layer that has a latent of its own a row per
// position, read by every layer that names it; per recurrent layer a state and, for the delta rule, the last inputs of
// its short convolutions.
//
// Launches of a decode step in bf16, after the sum and norm that the first projection of a sublayer does itself at one
// or two sequences: latent attention [query latent, latent, key part, gates], norms + rotation + cache, queries, absorb,
// attention, merge + values + gate, o; lightning [q, k, v, gate + silu], state, gated norm, o; delta rule [q, k, v,
// both low ranks, beta], everything up to the gated norm, o; feed-forward up + bias + relu^2, down + bias. A prompt pass
// has latent attention in its expanding form and takes the recurrences eight tokens at a time.
#include "lbk_mixers.cuh"
#include "lbk_runtime.cuh"

namespace lbk {

namespace {

enum class Mixer { Latent, Lightning, Delta };

struct DugulornLayer {
    Mixer type = Mixer::Latent;
    float *norm1 = nullptr, *norm2 = nullptr;
    DenseWeight in, o;                  // everything that reads the layer's input directly, stacked; the output
    // latent attention
    LatentShape lat;
    float scale = 1.0f;
    size_t source = 0;                  // the layer whose cache it reads (itself, or an earlier one)
    bool own = true;
    Rotation rot;
    DenseWeight uq, uk, uv, ukv;
    float *q_norm = nullptr, *kv_norm = nullptr;
    // recurrences
    size_t heads = 0, kv_heads = 0, dim = 0, vdim = 0, taps = 1;
    size_t a_at = 0, g_at = 0, b_at = 0;  // columns of the delta rule's low ranks and of beta in the rows of `in`
    float *decay = nullptr, *conv = nullptr, *a_log = nullptr, *dt_bias = nullptr, *mix_norm = nullptr;
    DenseWeight a2, g2;
    // feed-forward
    size_t ff = 0;
    DenseWeight up, down;
    float *up_bias = nullptr, *down_bias = nullptr;

    size_t out_width() const { return type == Mixer::Latent ? lat.heads * lat.vdim : heads * vdim; }
    size_t channels() const { return 2 * kv_heads * dim + heads * vdim; }
};

constexpr size_t kExpandRows = 32;      // prompt rows from which writing out keys and values pays
constexpr size_t kRecordRows = 1024;    // prompt rows whose records of a recurrence exist at a time

struct DugulornCache;

struct DugulornModel : Model {
    std::vector<DugulornLayer> layers;
    size_t width = 0;
    float eps = 0.0f;
    uint16_t *embed = nullptr;          // bf16 [vocab][width]
    DenseWeight head;                   // the same table
    float *embed_norm = nullptr, *final_norm = nullptr;
    int *zero = nullptr;
    bool all_expand = true;             // every latent layer can take the expanding form
    size_t elem() const { return compute == LBK_COMPUTE_F32 ? 4 : 2; }
    bool expands(size_t rows) const { return compute == LBK_COMPUTE_BF16 && all_expand && rows >= kExpandRows; }
    int make_cache(size_t batch, size_t capacity, std::unique_ptr<Cache> &out) override;
    int make_prefill_buffers(Cache *c, size_t rows) override;
    int enqueue_step(Cache *c, cudaStream_t st) override;
    int enqueue_rows(Cache *c, size_t seq, size_t n, cudaStream_t st) override;
    int enqueue_head(const float *rows, size_t n, float *logits, cudaStream_t st) override;
    struct Work;
    struct Pass;
    int make_work(std::vector<void *> &owner, Work &w, size_t rows, bool batch, size_t cap);
    int enqueue_tokens(DugulornCache *c, Work &w, const int32_t *tokens, size_t m, int seq, float *final_rows, cudaStream_t st);
    int enqueue_latent(const Pass &p, const DugulornLayer &l);
    int enqueue_recurrent(const Pass &p, const DugulornLayer &l, size_t li);
};

// Buffers of one pass over `rows` tokens, sized for the largest layer. Rows of the compute type have a pitch of a
// multiple of 64 values; what lies past a row's end is zero or a number another layer left there, and meets the
// zero columns of the weights.
struct DugulornModel::Work {
    float *x = nullptr, *x2 = nullptr, *y = nullptr;
    void *n = nullptr, *in = nullptr, *mid = nullptr, *h = nullptr;  // in: stacked projections of a recurrence; mid: a mixer's output
    float *z = nullptr;                                              // f32 projections: latent attention's, beta
    void *cq = nullptr, *q = nullptr, *ql = nullptr, *gate = nullptr;
    float *a = nullptr, *o = nullptr, *records = nullptr, *scratch = nullptr;
    size_t record_rows = 0;
};

struct DugulornCache : Cache {
    std::vector<void *> latent, ring;   // per layer: [b][cap][pitch]; [b][taps][channels]
    std::vector<float *> state;         // per layer: [b][heads][vdim][recur_pitch(dim)]
    DugulornModel::Work step_work, rows_work;
    float *final_rows = nullptr;
    // keys and values of one layer and sequence written out per head (prompt passes), grown as needed
    void *ek = nullptr, *ev = nullptr;
    size_t ek_bytes = 0, ev_bytes = 0, ecap = 0;
    ~DugulornCache() override {
        if (model) cudaSetDevice(model->ctx->device);
        cudaDeviceSynchronize();
        cudaFree(ek);
        cudaFree(ev);
    }
    int expand_room(const DugulornModel *m, size_t length);
};

// What every mixer of a pass needs. project: a projection of the layer's input rows.
struct DugulornModel::Pass {
    DugulornCache *c;
    Work &w;
    size_t m;
    int seq;
    const int *pos;
    cudaStream_t st;
};

int DugulornCache::expand_room(const DugulornModel *m, size_t length) {
    const size_t want = std::min(cap, (length + 255) / 256 * 256);
    size_t kb = 0, vb = 0;
    for (const DugulornLayer &l : m->layers)
        if (l.type == Mixer::Latent) {
            kb = std::max(kb, l.lat.heads * l.lat.dp() * 2);
            vb = std::max(vb, l.lat.heads * l.lat.vp() * 2);
        }
    if (kb == 0 || want <= ecap) return LBK_OK;
    const size_t rows = std::min(cap, std::max(want, ecap + ecap / 2));
    LBK_CUDA(cudaDeviceSynchronize());
    cudaFree(ek);
    cudaFree(ev);
    ek = ev = nullptr;
    ecap = 0;
    std::vector<void *> kept;           // freed by the destructor, not with the cache's other buffers
    LBK_TRY(dev_alloc(kept, kb * rows, &ek));
    LBK_TRY(dev_alloc(kept, vb * rows, &ev));
    LBK_CUDA(cudaMemset(ek, 0, kb * rows));  // padding of the head sizes meets zeros of the queries, but has to hold numbers
    LBK_CUDA(cudaMemset(ev, 0, vb * rows));
    LBK_CUDA(cudaDeviceSynchronize());
    ecap = rows;
    return LBK_OK;
}

int DugulornModel::make_work(std::vector<void *> &owner, Work &w, size_t rows, bool batch, size_t cap) {
    const size_t es = elem();
    // rows of the absorbing form: all of them, or the short passes only
    const size_t few = !batch && expands(rows) ? std::min(rows, kExpandRows - 1) : rows;
    size_t in = 0, mid = 0, h = 0, z = 0, cq = 0, q = 0, ql = 0, gate = 0, a = 0, o = 0, records = 0, scratch = 0;
    w.record_rows = std::min((rows + 7) / 8 * 8, kRecordRows);
    for (const DugulornLayer &l : layers) {
        mid = std::max(mid, dense_pitch(l.out_width()));
        h = std::max(h, dense_pitch(l.ff));
        if (l.type == Mixer::Latent) {
            z = std::max(z, l.in.rows);
            cq = std::max(cq, dense_pitch(l.lat.q_rank));
            q = std::max(q, l.lat.heads * l.lat.qp());
            ql = std::max(ql, l.lat.heads * l.lat.pitch());
            scratch = std::max(scratch, latent_scratch(ctx, few, l.lat, compute == LBK_COMPUTE_F32 ? 1 : latent_splits(cap)));
        } else {
            in = std::max(in, dense_pitch(l.in.rows));
            z = std::max(z, l.heads);
            o = std::max(o, l.heads * l.vdim);
            if (!batch) records = std::max(records, recur_record_floats(l.type == Mixer::Delta, w.record_rows, l.heads, l.dim, l.vdim));
            if (l.type == Mixer::Delta && !batch) {
                a = std::max(a, l.heads * l.dim);
                gate = std::max(gate, dense_pitch(l.heads * l.vdim));
            }
        }
    }
    struct { void **p; size_t bytes; } bufs[] = {
        {reinterpret_cast<void **>(&w.x), rows * width * 4}, {reinterpret_cast<void **>(&w.x2), rows * width * 4}, {reinterpret_cast<void **>(&w.y), rows * width * 4},
        {&w.n, rows * dense_pitch(width) * es}, {&w.in, rows * in * es}, {&w.mid, rows * mid * es}, {&w.h, rows * h * es},
        {reinterpret_cast<void **>(&w.z), rows * z * 4}, {&w.cq, rows * cq * es}, {&w.q, rows * q * es}, {&w.ql, few * ql * es}, {&w.gate, rows * gate * es},
        {reinterpret_cast<void **>(&w.a), rows * a * 4}, {reinterpret_cast<void **>(&w.o), rows * o * 4}, {reinterpret_cast<void **>(&w.records), records * 4},
        {reinterpret_cast<void **>(&w.scratch), scratch * 4}};
    for (auto &b : bufs) {
        LBK_TRY(dev_alloc(owner, b.bytes, b.p));
        LBK_CUDA(cudaMemset(*b.p, 0, b.bytes ? b.bytes : 16));
    }
    LBK_CUDA(cudaDeviceSynchronize());
    return LBK_OK;
}

int DugulornModel::make_cache(size_t batch, size_t capacity, std::unique_ptr<Cache> &out) {
    DugulornCache *c = new DugulornCache();
    out.reset(c);
    if (capacity == 0) capacity = 4096;  // positions have no limit of their own
    if (capacity > (1u << 30)) return fail(LBK_ERR_UNSUPPORTED, "a cache of %zu positions", capacity);
    c->cap = capacity;
    for (const DugulornLayer &l : layers) {
        void *latent = nullptr, *ring = nullptr, *state = nullptr;
        if (l.type == Mixer::Latent && l.own) {
            const size_t bytes = batch * capacity * l.lat.pitch() * elem();
            LBK_TRY(dev_alloc(c->device_allocs, bytes, &latent));
            LBK_CUDA(cudaMemset(latent, 0, bytes));  // the padding of a row stays zero
        } else if (l.type != Mixer::Latent) {
            // a sequence at position 0 starts from zeros whatever these hold
            LBK_TRY(dev_alloc(c->device_allocs, batch * l.heads * l.vdim * recur_pitch(l.dim) * 4, &state));
            if (l.type == Mixer::Delta) LBK_TRY(dev_alloc(c->device_allocs, batch * l.taps * l.channels() * elem(), &ring));
        }
        c->latent.push_back(latent);
        c->ring.push_back(ring);
        c->state.push_back(static_cast<float *>(state));
    }
    LBK_TRY(make_work(c->device_allocs, c->step_work, batch, true, capacity));
    return dev_alloc(c->device_allocs, batch * width * 4, reinterpret_cast<void **>(&c->final_rows));
}

int DugulornModel::make_prefill_buffers(Cache *cache, size_t rows) {
    DugulornCache *c = static_cast<DugulornCache *>(cache);
    return make_work(c->pf_allocs, c->rows_work, rows, false, c->cap);
}

// From the stacked projections in w.z to w.mid.
int DugulornModel::enqueue_latent(const Pass &p, const DugulornLayer &l) {
    Work &w = p.w;
    const LatentShape &s = l.lat;
    const long ldz = static_cast<long>(l.in.rows);
    LatentPrepCall pc;
    pc.compute = compute;
    pc.s = s;
    pc.z = w.z;
    pc.ldz = ldz;
    pc.rows = p.m;
    pc.rows_of_seq = p.seq;
    pc.pos = p.pos;
    pc.cap = p.c->cap;
    pc.q_norm = l.q_norm;
    pc.kv_norm = l.kv_norm;
    pc.eps = eps;
    pc.rot = l.rot;
    pc.cq = w.cq;
    pc.ldq = static_cast<long>(l.uq.pitch);
    pc.cache = l.own ? p.c->latent[l.source] : nullptr;
    LBK_TRY(launch_latent_prep(ctx, pc, p.st));
    DenseCall d;
    d.compute = compute;
    d.m = p.m;
    d.x = w.cq;
    d.ldx = static_cast<long>(l.uq.pitch);
    d.w = l.uq;
    d.out_rows = l.uq.rows;
    d.epi.kind = kEpiQkv;
    d.epi.out = w.q;
    d.epi.ld = static_cast<long>(s.heads * s.qp());
    d.epi.q_rows = static_cast<int>(l.uq.rows);
    d.epi.dim = static_cast<int>(s.dim + s.rot_dim);
    d.epi.dimp = static_cast<int>(s.qp());
    d.epi.q_split = static_cast<int>(s.dim);
    d.epi.q_gap = static_cast<int>(s.dp() - s.dim);
    LBK_TRY(launch_dense(ctx, d, p.st));
    LatentAttnCall a;
    a.compute = compute;
    a.s = s;
    a.q = w.q;
    a.rows = p.m;
    a.rows_of_seq = p.seq;
    a.pos = p.pos;
    a.cap = p.c->cap;
    a.cache = p.c->latent[l.source];
    a.uk = l.uk;
    a.uv = l.uv;
    a.ukv = l.ukv;
    a.scale = l.scale;
    a.rot = l.rot;
    a.gate = w.z + (l.in.rows - s.heads);
    a.ldg = ldz;
    a.out = w.mid;
    a.ldo = static_cast<long>(l.o.pitch);
    if (p.seq >= 0 && expands(p.m)) {
        a.length = p.c->lens[static_cast<size_t>(p.seq)] + p.m;
        a.ek = p.c->ek;
        a.ev = p.c->ev;
        a.ecap = p.c->ecap;
        a.zero = zero;
        return launch_latent_expanded(ctx, a, p.st);
    }
    a.ql = w.ql;
    a.scratch = w.scratch;
    a.splits = latent_splits(p.c->cap);
    return launch_latent_absorbed(ctx, a, p.st);
}

// From the stacked projections in w.in (and beta's logits in w.z) to w.mid.
int DugulornModel::enqueue_recurrent(const Pass &p, const DugulornLayer &l, size_t li) {
    Work &w = p.w;
    const bool delta = l.type == Mixer::Delta;
    const long ldin = static_cast<long>(dense_pitch(l.in.rows));
    const size_t hv = l.heads * l.vdim, qk = l.kv_heads * l.dim;
    RecurCall r;
    GatedNormCall g;
    if (delta && p.seq < 0) {
        r.a2 = l.a2;
        r.g2 = l.g2;
        r.a_at = static_cast<int>(l.a_at);
        r.g_at = static_cast<int>(l.g_at);
        r.norm_w = l.mix_norm;
        r.eps = eps;
        r.out = w.mid;
        r.ldo = static_cast<long>(l.o.pitch);
    } else if (delta) {
        DenseCall d;
        d.compute = compute;
        d.m = p.m;
        d.ldx = ldin;
        d.x = static_cast<const char *>(w.in) + l.a_at * elem();
        d.w = l.a2;
        d.out_rows = l.a2.rows;
        d.epi.kind = kEpiF32;
        d.epi.out = w.a;
        d.epi.ld = static_cast<long>(l.a2.rows);
        LBK_TRY(launch_dense(ctx, d, p.st));
        d.x = static_cast<const char *>(w.in) + l.g_at * elem();
        d.w = l.g2;
        d.out_rows = l.g2.rows;
        d.epi.kind = kEpiElem;
        d.epi.out = w.gate;
        d.epi.ld = static_cast<long>(dense_pitch(hv));
        LBK_TRY(launch_dense(ctx, d, p.st));
        g.gate = w.gate;
        g.ldg = static_cast<long>(dense_pitch(hv));
        g.group = l.vdim;
    } else {
        g.gate = static_cast<const char *>(w.in) + (2 * qk + hv) * elem();
        g.ldg = ldin;
        g.group = hv;
    }
    r.compute = compute;
    r.delta = delta;
    r.heads = l.heads;
    r.kv_heads = l.kv_heads;
    r.dim = l.dim;
    r.vdim = l.vdim;
    r.x = w.in;
    r.ldx = ldin;
    r.q_at = 0;
    r.k_at = static_cast<int>(qk);
    r.v_at = static_cast<int>(2 * qk);
    r.rows = p.m;
    r.rows_of_seq = p.seq;
    r.pos = p.pos;
    r.active = p.c->active;
    r.cap = p.c->cap;
    r.decay = l.decay;
    r.taps = static_cast<int>(l.taps);
    r.conv = l.conv;
    r.ring = p.c->ring[li];
    r.a = w.a;
    r.lda = static_cast<long>(l.heads * l.dim);
    r.a_log = l.a_log;
    r.dt_bias = l.dt_bias;
    r.b = w.z;
    r.ldb = static_cast<long>(l.heads);
    r.state = p.c->state[li];
    r.records = w.records;
    r.record_rows = w.record_rows;
    r.o = w.o;
    LBK_TRY(launch_recurrence(ctx, r, p.st));
    if (r.out) return LBK_OK;
    g.compute = compute;
    g.o = w.o;
    g.rows = p.m;
    g.n = hv;
    g.w = l.mix_norm;
    g.eps = eps;
    g.out = w.mid;
    g.ldo = static_cast<long>(l.o.pitch);
    return launch_gated_norm(ctx, g, p.st);
}

// `m` tokens through all layers: consecutive positions of sequence `seq`, or (seq < 0) one token of each sequence.
int DugulornModel::enqueue_tokens(DugulornCache *c, Work &w, const int32_t *tokens, size_t m, int seq, float *final_rows, cudaStream_t st) {
    const bool fuse = compute == LBK_COMPUTE_BF16 && dense_pre_supported(m, width);  // sums and norms run inside the projection behind them
    const long npitch = static_cast<long>(dense_pitch(width));
    const Pass pass{c, w, m, seq, c->pos + (seq >= 0 ? seq : 0), st};
    LBK_TRY(lbk_embed_bf16(reinterpret_cast<lbk_ctx *>(ctx), embed, tokens, m, width, w.x, st));
    float *x = w.x, *x2 = w.x2;
    // what the last sublayer still owes the residual: its output rows and the norm in front of the sum
    const float *y = nullptr, *w_post = nullptr;

    auto norm_rows = [&](const float *w_next, void *out_e, float *out_f) -> int {
        NormCall n;
        n.compute = compute;
        n.rms = true;
        n.x = x;
        n.y = y;
        n.w_post = w_post;
        n.w = w_next;
        n.rows = m;
        n.n = width;
        n.eps = eps;
        n.out_e = out_e;
        n.lde = npitch;
        n.out_f = out_f;
        y = nullptr;
        return launch_sandwich_norm(ctx, n, st);
    };
    // the projection `d` of the residual
    auto project = [&](DenseCall &d) -> int {
        d.compute = compute;
        d.m = m;
        d.x = w.n;
        d.ldx = npitch;
        if (y && !fuse) LBK_TRY(norm_rows(nullptr, w.n, nullptr));
        if (!y) return launch_dense(ctx, d, st);
        d.pre.mode = kPreAddNorm;
        d.pre.rms = true;
        d.pre.x = x;
        d.pre.y = y;
        d.pre.w_post = w_post;
        d.pre.xout = x2;
        d.pre.eps = eps;
        y = nullptr;
        std::swap(x, x2);
        return launch_dense(ctx, d, st);
    };
    // the last projection of a sublayer: its rows wait for their norm
    auto leave = [&](const void *in, const DenseWeight &wt, const float *bias, const float *norm) -> int {
        DenseCall d;
        d.compute = compute;
        d.m = m;
        d.x = in;
        d.ldx = static_cast<long>(wt.pitch);
        d.w = wt;
        d.out_rows = wt.rows;
        d.epi.kind = kEpiF32;
        d.epi.bias = bias;
        d.epi.out = w.y;
        d.epi.ld = static_cast<long>(wt.rows);
        y = w.y;
        w_post = norm;
        return launch_dense(ctx, d, st);
    };

    LBK_TRY(norm_rows(embed_norm, w.n, x));
    for (size_t li = 0; li < layers.size(); ++li) {
        const DugulornLayer &l = layers[li];
        DenseCall d;
        d.w = l.in;
        d.out_rows = l.in.rows;
        if (l.type == Mixer::Latent) {
            d.epi.kind = kEpiF32;
            d.epi.out = w.z;
            d.epi.ld = static_cast<long>(l.in.rows);
            LBK_TRY(project(d));
            LBK_TRY(enqueue_latent(pass, l));
        } else {
            d.epi.kind = kEpiElem;
            d.epi.out = w.in;
            d.epi.ld = static_cast<long>(dense_pitch(l.in.rows));
            if (l.type == Mixer::Lightning) {
                d.epi.act = kActSilu;
                d.epi.act_rows = static_cast<int>(l.channels());
            } else {
                d.epi.f32_from = static_cast<int>(l.b_at);
                d.epi.out2 = w.z;
                d.epi.ld2 = static_cast<long>(l.heads);
            }
            LBK_TRY(project(d));
            LBK_TRY(enqueue_recurrent(pass, l, li));
        }
        LBK_TRY(leave(w.mid, l.o, nullptr, l.norm1));
        if (l.ff) {
            DenseCall u;
            u.w = l.up;
            u.out_rows = l.ff;
            u.epi.kind = kEpiElem;
            u.epi.act = kActRelu2;
            u.epi.bias = l.up_bias;
            u.epi.out = w.h;
            u.epi.ld = static_cast<long>(l.down.pitch);
            LBK_TRY(project(u));
            LBK_TRY(leave(w.h, l.down, l.down_bias, l.norm2));
        }
    }
    return norm_rows(final_norm, nullptr, final_rows);
}

int DugulornModel::enqueue_step(Cache *cache, cudaStream_t st) {
    DugulornCache *c = static_cast<DugulornCache *>(cache);
    LBK_TRY(enqueue_tokens(c, c->step_work, c->tokens, c->b, -1, c->final_rows, st));
    return enqueue_head(c->final_rows, c->b, c->logits, st);
}

int DugulornModel::enqueue_rows(Cache *cache, size_t seq, size_t n, cudaStream_t st) {
    DugulornCache *c = static_cast<DugulornCache *>(cache);
    if (expands(n)) LBK_TRY(c->expand_room(this, c->lens[seq] + n));
    return enqueue_tokens(c, c->rows_work, c->pf_tokens, n, static_cast<int>(seq), c->pf_n, st);
}

int DugulornModel::enqueue_head(const float *rows, size_t n, float *logits, cudaStream_t st) {
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
bool json_number(const Json *j, double *out) {
    if (!j || j->kind != Json::Num) return false;
    *out = j->num;
    return true;
}

struct LayerReader {
    const std::string &dir;
    DugulornModel *m;
    WeightLoader &ld;
    size_t i;
    std::string p;        // "l<i>."
    const Json &mx;
    DugulornLayer &l;

    int bad(const char *what) const { return fail(LBK_ERR_INVALID, "%s/config.json: layer %zu: %s is missing or inconsistent", dir.c_str(), i, what); }

    int rotation() {
        const Json *rot = mx.get("rot");
        double base = 0.0;
        size_t dims = 0;
        if (!rot || rot->kind != Json::Obj || !json_number(rot->get("base"), &base) || base <= 0.0 || !json_positive(rot->get("dims"), &dims) || dims != l.lat.rot_dim || dims % 2)
            return bad("mixer.rot");
        YarnScaling y;
        const Json *sc = rot->get("scaling");
        if (sc && sc->kind == Json::Obj) {
            y.on = true;
            if (!json_number(sc->get("factor"), &y.factor) || !json_number(sc->get("original"), &y.original) || !json_number(sc->get("fast"), &y.fast) ||
                !json_number(sc->get("slow"), &y.slow) || y.factor <= 0.0 || y.original <= 0.0 || y.fast <= 0.0 || y.slow <= 0.0)
                return bad("mixer.rot.scaling");
        }
        std::vector<double> freq(dims / 2);
        rotation_frequencies(dims, base, y, freq.data(), &l.rot.factor);
        l.rot.dims = static_cast<int>(dims);
        double *dev = nullptr;
        LBK_TRY(dev_alloc(m->device_allocs, freq.size() * sizeof(double), reinterpret_cast<void **>(&dev)));
        LBK_CUDA(cudaMemcpy(dev, freq.data(), freq.size() * sizeof(double), cudaMemcpyHostToDevice));
        l.rot.freq = dev;
        return LBK_OK;
    }

    int latent() {
        l.type = Mixer::Latent;
        LatentShape &s = l.lat;
        double scale = 0.0;
        if (!json_positive(mx.get("heads"), &s.heads) || !json_positive(mx.get("dim"), &s.dim) || !json_positive(mx.get("rot_dim"), &s.rot_dim) ||
            !json_positive(mx.get("vdim"), &s.vdim) || !json_positive(mx.get("kv_rank"), &s.kv_rank) || !json_number(mx.get("scale"), &scale))
            return bad("heads, dim, rot_dim, vdim, kv_rank or scale");
        l.scale = static_cast<float>(scale);
        size_t cols = 0;
        LBK_TRY(ld.shape(p + "mix.dq", &s.q_rank, &cols));
        LBK_TRY(rotation());
        const Json *from = mx.get("kv_from");
        l.source = i;
        if (from && from->kind == Json::Num) {
            l.own = false;
            l.source = from->num >= 0 && from->num < static_cast<double>(i) ? static_cast<size_t>(from->num) : i;
            if (l.source == i) return bad("mixer.kv_from (an earlier layer)");
            const DugulornLayer &src = m->layers[l.source];
            if (src.type != Mixer::Latent || !src.own || src.lat.kv_rank != s.kv_rank || src.lat.rot_dim != s.rot_dim) return bad("mixer.kv_from (a latent of the same sizes)");
        }
        if (m->compute == LBK_COMPUTE_BF16 && !latent_absorb_supported(s))
            return fail(LBK_ERR_UNSUPPORTED, "layer %zu: in bf16 latents of at most 512 values, rotated parts of at most 128", i);
        m->all_expand = m->all_expand && latent_expand_supported(s);
        std::vector<std::string> in{p + "mix.dq"};
        std::vector<size_t> rows{s.q_rank};
        if (l.own) {
            in.push_back(p + "mix.dkv");
            rows.push_back(s.kv_rank + s.rot_dim);
            LBK_TRY(ld.vec(p + "mix.dkv.norm", s.kv_rank, &l.kv_norm));
        }
        in.push_back(p + "mix.g");
        rows.push_back(s.heads);
        LBK_TRY(ld.stack(in, rows, m->width, &l.in));
        LBK_TRY(ld.vec(p + "mix.dq.norm", s.q_rank, &l.q_norm));
        LBK_TRY(ld.stack({p + "mix.uq"}, {s.heads * (s.dim + s.rot_dim)}, s.q_rank, &l.uq));
        LBK_TRY(ld.stack({p + "mix.uk", p + "mix.uv"}, {s.heads * s.dim, s.heads * s.vdim}, s.kv_rank, &l.ukv));
        l.uk = l.uv = l.ukv;
        l.uk.rows = s.heads * s.dim;
        l.uv.rows = s.heads * s.vdim;
        l.uv.w = l.ukv.w + l.uk.rows * l.ukv.pitch;
        return LBK_OK;
    }

    int sizes() {
        if (!json_positive(mx.get("heads"), &l.heads) || !json_positive(mx.get("dim"), &l.dim) || !json_positive(mx.get("vdim"), &l.vdim)) return bad("heads, dim or vdim");
        if (l.dim > kRecurMaxDim || l.vdim > 1024) return fail(LBK_ERR_UNSUPPORTED, "layer %zu: key heads of at most %zu dimensions, value heads of at most 1024", i, kRecurMaxDim);
        return LBK_OK;
    }

    int lightning() {
        l.type = Mixer::Lightning;
        LBK_TRY(sizes());
        l.kv_heads = l.heads;
        const Json *decay = mx.get("decay");
        if (!decay || decay->kind != Json::Arr || decay->arr.size() != l.heads) return bad("mixer.decay (one per head)");
        std::vector<float> v;
        for (const Json &d : decay->arr) {
            if (d.kind != Json::Num) return bad("mixer.decay (one per head)");
            v.push_back(static_cast<float>(d.num));
        }
        LBK_TRY(ld.floats(v, &l.decay));
        const size_t qk = l.heads * l.dim, hv = l.heads * l.vdim;
        LBK_TRY(ld.stack({p + "mix.q", p + "mix.k", p + "mix.v", p + "mix.g"}, {qk, qk, hv, hv}, m->width, &l.in));
        return ld.vec(p + "mix.norm", hv, &l.mix_norm);
    }

    int delta() {
        l.type = Mixer::Delta;
        LBK_TRY(sizes());
        if (!json_positive(mx.get("kv_heads"), &l.kv_heads) || l.heads % l.kv_heads) return bad("kv_heads");
        const size_t qk = l.kv_heads * l.dim, hv = l.heads * l.vdim;
        size_t rows = 0, cols = 0, ra = 0, rg = 0;
        LBK_TRY(ld.shape(p + "mix.q.conv", &rows, &l.taps));
        if (mx.get("conv") && (!json_positive(mx.get("conv"), &cols) || cols != l.taps)) return bad("mixer.conv");
        // q, k, v, then the low ranks from a multiple of 64 columns on (each is the operand of a projection), then beta
        LBK_TRY(ld.shape(p + "mix.a1", &ra, &cols));
        LBK_TRY(ld.shape(p + "mix.g1", &rg, &cols));
        const size_t ch = l.channels();
        l.a_at = dense_pitch(ch);
        l.g_at = l.a_at + dense_pitch(ra);
        l.b_at = l.g_at + dense_pitch(rg);
        LBK_TRY(ld.stack({p + "mix.q", p + "mix.k", p + "mix.v", "", p + "mix.a1", "", p + "mix.g1", "", p + "mix.b"},
                         {qk, qk, hv, l.a_at - ch, ra, l.g_at - l.a_at - ra, rg, l.b_at - l.g_at - rg, l.heads}, m->width, &l.in));
        LBK_TRY(ld.stack({p + "mix.a2"}, {l.heads * l.dim}, ra, &l.a2));
        LBK_TRY(ld.stack({p + "mix.g2"}, {hv}, rg, &l.g2));
        // [channels][taps] in the file, [taps][channels] on the device
        std::vector<float> conv(ch * l.taps), part;
        size_t at = 0;
        const struct { const char *name; size_t n; } parts[3] = {{"mix.q.conv", qk}, {"mix.k.conv", qk}, {"mix.v.conv", hv}};
        for (const auto &c : parts) {
            LBK_TRY(ld.read(p + c.name, c.n * l.taps, part));
            for (size_t k = 0; k < c.n; ++k)
                for (size_t j = 0; j < l.taps; ++j) conv[j * ch + at + k] = part[k * l.taps + j];
            at += c.n;
        }
        LBK_TRY(ld.floats(conv, &l.conv));
        LBK_TRY(ld.vec(p + "mix.A_log", l.heads, &l.a_log));
        LBK_TRY(ld.vec(p + "mix.dt_bias", l.heads * l.dim, &l.dt_bias));
        return ld.vec(p + "mix.norm", l.vdim, &l.mix_norm);
    }

    int feed_forward(const Json &mlp) {
        const Json *kind = mlp.get("kind");
        if (!kind || kind->kind != Json::Str || kind->str != "dense")
            return fail(LBK_ERR_UNSUPPORTED, "%s/config.json: layer %zu: unknown feed-forward \"%s\"", dir.c_str(), i, kind && kind->kind == Json::Str ? kind->str.c_str() : "");
        size_t cols = 0;
        LBK_TRY(ld.shape(p + "mlp.up", &l.ff, &cols));
        LBK_TRY(ld.vec(p + "norm2", m->width, &l.norm2, 1.0f));
        LBK_TRY(ld.stack({p + "mlp.up"}, {l.ff}, m->width, &l.up));
        LBK_TRY(ld.stack({p + "mlp.down"}, {m->width}, l.ff, &l.down));
        LBK_TRY(ld.vec(p + "mlp.up.b", l.ff, &l.up_bias));
        return ld.vec(p + "mlp.down.b", m->width, &l.down_bias);
    }
};

int load_dugulorn(Ctx *ctx, const std::string &dir, const Json &cj, int compute, int, int world, std::unique_ptr<Model> &out) {
    if (world > 1) return fail(LBK_ERR_UNSUPPORTED, "the Dugulorn family is not sharded over ranks");
    DugulornModel *m = new DugulornModel();
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
    size_t vocab = 0, width = 0, cv = 0, cw = 0;
    LBK_TRY(ld.shape("embed", &vocab, &width));
    if (!vocab || !width || (json_positive(cj.get("vocab"), &cv) && cv != vocab) || (json_positive(cj.get("width"), &cw) && cw != width))
        return fail(LBK_ERR_SHAPE, "%s: embed is [%zu, %zu]; config.json says vocab %zu, width %zu", tf.path.c_str(), vocab, width, cv, cw);
    m->width = width;
    LBK_TRY(ld.table("embed", vocab, width, &m->embed));
    m->head = DenseWeight{m->embed, vocab, width, width};
    LBK_TRY(ld.vec("embed.norm", width, &m->embed_norm, 1.0f));
    LBK_TRY(ld.vec("final.norm", width, &m->final_norm, 1.0f));
    LBK_TRY(dev_alloc(m->device_allocs, 4, reinterpret_cast<void **>(&m->zero)));
    LBK_CUDA(cudaMemset(m->zero, 0, 4));
    size_t first_ff = 0;
    m->layers.reserve(layers->arr.size());
    for (size_t i = 0; i < layers->arr.size(); ++i) {
        const Json &lj = layers->arr[i];
        const Json *type = lj.get("type"), *mx = lj.get("mixer"), *mlp = lj.get("mlp");
        const std::string ts = type && type->kind == Json::Str ? type->str : "";
        if (!mx || mx->kind != Json::Obj) return fail(LBK_ERR_INVALID, "%s/config.json: layer %zu has no mixer", dir.c_str(), i);
        DugulornLayer l;
        LayerReader r{dir, m, ld, i, "l" + std::to_string(i) + ".", *mx, l};
        LBK_TRY(ld.vec(r.p + "norm1", width, &l.norm1, 1.0f));
        if (ts == "latent_attention") LBK_TRY(r.latent());
        else if (ts == "lightning") LBK_TRY(r.lightning());
        else if (ts == "channel_delta") LBK_TRY(r.delta());
        else return fail(LBK_ERR_UNSUPPORTED, "%s/config.json: layer %zu: unknown mixer \"%s\"", dir.c_str(), i, ts.c_str());
        LBK_TRY(ld.stack({r.p + "mix.o"}, {width}, l.out_width(), &l.o));
        if (mlp && mlp->kind == Json::Obj) {
            LBK_TRY(r.feed_forward(*mlp));
            if (!first_ff) first_ff = l.ff;
        }
        m->layers.push_back(l);
    }
    LBK_CUDA(cudaStreamSynchronize(ctx->own_stream));  // the staging buffers go away now
    LBK_CUDA(cudaDeviceSynchronize());
    const DugulornLayer &front = m->layers[0];
    lbk_model_config &cfg = m->cfg;
    cfg.hidden_size = width;
    cfg.intermediate_size = first_ff;
    cfg.num_attention_heads = front.type == Mixer::Latent ? front.lat.heads : front.heads;
    cfg.num_key_value_heads = front.type == Mixer::Latent ? 1 : front.kv_heads;
    cfg.num_hidden_layers = m->layers.size();
    cfg.vocab_size = vocab;
    cfg.rms_norm_eps = m->eps;
    m->stats.bytes_read = tf.sg.bytes_read;
    m->stats.bytes_to_device = tf.sg.bytes_to_device;
    return LBK_OK;
}

const FamilyRegistrar kDugulorn("Dugulorn", load_dugulorn);

}  // namespace

}  // namespace lbk
