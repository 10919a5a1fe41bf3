// The decoder models as a native runtime behind the C ABI, for hosts that want lb-model's
// `BitNet::{load, new_cache, forward}` (crates/lb-model/src/model.rs:149-232, 234-236, 305-374) without a
// tensor framework in between: the registry of model families, the checkpoint file, the cache's slots and
// positions, the recorded decode step, prompt passes, and the batcher. What a family's step consists of is
// in its own file (lbk_bitnet.cu, lbk_pefolix.cu, lbk_dugulorn.cu).
//
// A call with several tokens of one sequence (a prompt, or a portion of one) sends up to 4096 rows at a time
// through the projections. One decode step is recorded into a CUDA graph the first time a cache is used and
// replayed afterwards (the positions live in device memory).
#include <deque>

#include "lbk_runtime.cuh"

namespace lbk {

Cache::~Cache() {
    if (model) cudaSetDevice(model->ctx->device);
    cudaDeviceSynchronize();
    if (step) cudaGraphExecDestroy(step);
    for (void *p : device_allocs) cudaFree(p);
    for (void *p : pf_allocs) cudaFree(p);
}

Model::~Model() {
    if (ctx) cudaSetDevice(ctx->device);
    cudaDeviceSynchronize();
    for (void *p : device_allocs) cudaFree(p);
}

// ---- families -----------------------------------------------------------------------------------
namespace {
std::map<std::string, LoadFn> &families() {
    static std::map<std::string, LoadFn> f;
    return f;
}
}  // namespace

FamilyRegistrar::FamilyRegistrar(const char *architecture, LoadFn load) { families()[architecture] = load; }

// ---- safetensors --------------------------------------------------------------------------------
int TensorFile::open_file(const std::string &file, cudaStream_t stream) {
    path = file;
    sg.fd = open(path.c_str(), O_RDONLY);
    if (sg.fd < 0) return fail(LBK_ERR_INVALID, "cannot open %s", path.c_str());
    struct stat sb;
    if (fstat(sg.fd, &sb) != 0) return fail(LBK_ERR_INVALID, "cannot stat %s", path.c_str());
    sg.file_size = static_cast<size_t>(sb.st_size);
    unsigned char lenb[8];
    if (sg.file_size < 8 || pread(sg.fd, lenb, 8, 0) != 8) return fail(LBK_ERR_INVALID, "%s: truncated", path.c_str());
    uint64_t hlen = 0;
    for (int i = 7; i >= 0; --i) hlen = (hlen << 8) | lenb[i];
    if (hlen == 0 || hlen > (100u << 20)) return fail(LBK_ERR_INVALID, "%s: implausible header length %llu", path.c_str(), static_cast<unsigned long long>(hlen));
    if (8 + hlen > sg.file_size) return fail(LBK_ERR_INVALID, "%s: truncated header", path.c_str());
    std::string header(hlen, '\0');
    if (pread(sg.fd, &header[0], hlen, 8) != static_cast<ssize_t>(hlen)) return fail(LBK_ERR_INVALID, "%s: truncated header", path.c_str());
    Json hj;
    if (!parse_json(header, hj) || hj.kind != Json::Obj) return fail(LBK_ERR_INVALID, "%s: header is not a JSON object", path.c_str());
    const Json *meta = hj.get("__metadata__");
    const Json *fmt = meta ? meta->get("format") : nullptr;
    if (fmt && fmt->kind == Json::Str) format = fmt->str;
    for (const auto &kv : hj.obj) {
        if (kv.first == "__metadata__") continue;
        const Json &t = kv.second;
        const Json *dt = t.get("dtype"), *sh = t.get("shape"), *off = t.get("data_offsets");
        if (!dt || dt->kind != Json::Str || !sh || sh->kind != Json::Arr || !off || off->kind != Json::Arr || off->arr.size() != 2)
            return fail(LBK_ERR_INVALID, "%s: malformed entry %s", path.c_str(), kv.first.c_str());
        TensorEntry e;
        e.dtype = dt->str;
        for (const Json &d : sh->arr) e.shape.push_back(static_cast<size_t>(d.num));
        e.begin = static_cast<size_t>(off->arr[0].num);
        e.end = static_cast<size_t>(off->arr[1].num);
        if (e.end < e.begin) return fail(LBK_ERR_INVALID, "%s: malformed offsets of %s", path.c_str(), kv.first.c_str());
        entries[kv.first] = e;
    }
    sg.data0 = static_cast<size_t>(8 + hlen);
    return sg.init(stream);
}

int TensorFile::find(const std::string &name, const char *dtype, size_t elems, size_t elem_bytes, const TensorEntry **e_out) const {
    auto it = entries.find(name);
    if (it == entries.end()) return fail(LBK_ERR_INVALID, "%s: tensor %s is missing", path.c_str(), name.c_str());
    const TensorEntry &e = it->second;
    size_t n = 1;
    for (size_t d : e.shape) n *= d;
    if (e.dtype != dtype || n != elems || e.end - e.begin != elems * elem_bytes)
        return fail(LBK_ERR_SHAPE, "%s: %s has dtype %s and %zu elements, expected %s and %zu", path.c_str(), name.c_str(), e.dtype.c_str(), n, dtype, elems);
    if (sg.data0 + e.end > sg.file_size)
        return fail(LBK_ERR_INVALID, "%s is truncated: %s ends at byte %zu, the file has %zu", path.c_str(), name.c_str(), sg.data0 + e.end, sg.file_size);
    *e_out = &e;
    return LBK_OK;
}

int WeightLoader::shape(const std::string &name, size_t *rows, size_t *cols) const {
    const auto it = tf.entries.find(name);
    if (it == tf.entries.end()) return fail(LBK_ERR_INVALID, "%s: tensor %s is missing", tf.path.c_str(), name.c_str());
    if (it->second.shape.size() != 2) return fail(LBK_ERR_SHAPE, "%s: %s is not a matrix", tf.path.c_str(), name.c_str());
    *rows = it->second.shape[0];
    *cols = it->second.shape[1];
    return LBK_OK;
}

int WeightLoader::read(const std::string &name, size_t n, std::vector<float> &f) {
    const TensorEntry *e;
    LBK_TRY(tf.find(name, "BF16", n, 2, &e));
    std::vector<uint16_t> raw(n);
    if (pread(tf.sg.fd, raw.data(), n * 2, static_cast<off_t>(tf.sg.data0 + e->begin)) != static_cast<ssize_t>(n * 2))
        return fail(LBK_ERR_INVALID, "cannot read %s", name.c_str());
    f.resize(n);
    for (size_t i = 0; i < n; ++i) {
        const uint32_t bits = static_cast<uint32_t>(raw[i]) << 16;
        memcpy(&f[i], &bits, 4);
    }
    tf.sg.bytes_read += n * 2;
    return LBK_OK;
}

int WeightLoader::vec(const std::string &name, size_t n, float **out, float add) {
    std::vector<float> f;
    LBK_TRY(read(name, n, f));
    for (float &v : f) v += add;
    return floats(f, out);
}

int WeightLoader::floats(const std::vector<float> &v, float **out) {
    LBK_TRY(dev_alloc(owner, v.size() * 4, reinterpret_cast<void **>(out)));
    LBK_CUDA(cudaMemcpy(*out, v.data(), v.size() * 4, cudaMemcpyHostToDevice));
    tf.sg.bytes_to_device += v.size() * 4;
    return LBK_OK;
}

int WeightLoader::stack(const std::vector<std::string> &names, const std::vector<size_t> &rows, size_t cols, DenseWeight *out) {
    size_t total = 0;
    bool zeros = false;
    for (size_t i = 0; i < rows.size(); ++i) {
        total += rows[i];
        zeros = zeros || names[i].empty();
    }
    const size_t pitch = dense_pitch(cols);
    uint16_t *dev = nullptr;
    LBK_TRY(dev_alloc(owner, total * pitch * 2, reinterpret_cast<void **>(&dev)));
    if (pitch != cols || zeros) LBK_CUDA(cudaMemsetAsync(dev, 0, total * pitch * 2, ctx->own_stream));
    size_t at = 0;
    for (size_t i = 0; i < names.size(); ++i) {
        if (!names[i].empty()) {
            const TensorEntry *e;
            LBK_TRY(tf.find(names[i], "BF16", rows[i] * cols, 2, &e));
            LBK_TRY(tf.sg.copy_rows(e->begin, rows[i], cols * 2, dev + at * pitch, pitch * 2, names[i].c_str()));
        }
        at += rows[i];
    }
    *out = DenseWeight{dev, total, cols, pitch};
    return LBK_OK;
}

int WeightLoader::table(const std::string &name, size_t rows, size_t cols, uint16_t **out) {
    const TensorEntry *e;
    LBK_TRY(tf.find(name, "BF16", rows * cols, 2, &e));
    LBK_TRY(dev_alloc(owner, rows * cols * 2, reinterpret_cast<void **>(out)));
    return tf.sg.copy_linear(e->begin, rows * cols * 2, *out, name.c_str());
}

bool json_positive(const Json *j, size_t *out) {
    if (!j || j->kind != Json::Num || j->num < 1 || j->num > 1e9 || j->num != std::floor(j->num)) return false;
    *out = static_cast<size_t>(j->num);
    return true;
}

// Continuous batching over one cache of `slots` sequences: what the reference's server would need in
// front of a batched decode step (its worker serves one request at a time,
// crates/lb-server/src/main.rs:92-166). Requests wait in a queue; a free slot takes the next one
// (its prompt goes through the prompt pass into that slot); every step advances all occupied slots
// by one greedy token (sample.rs:17-25) with the recorded decode step; a finished request frees
// its slot at once.
struct Request {
    uint64_t id = 0;
    std::vector<uint32_t> prompt, out;
    size_t max_new = 0;
    int32_t eos = -1;
    bool done = false;
    int slot = -1;
};

struct Batcher {
    Model *model = nullptr;
    Cache *cache = nullptr;
    std::deque<uint64_t> queue;
    std::map<uint64_t, Request> reqs;
    std::vector<uint64_t> slot_req;  // 0: the slot is free
    uint64_t next_id = 1;
};

namespace {

constexpr size_t kLogitRows = 128;      // rows of logits staged on the device at a time

// Work buffers for prompt passes of up to `rows` rows, allocated for the rows a prompt really has (more rows
// fill the GEMM's tile rounds better: a 4032-token prompt at 2B4T shapes takes 41.3 ms at 1024 rows a pass,
// 34.8 at 2048, 30.6 at 4096).
int ensure_prefill_buffers(Model *m, Cache *c, size_t rows) {
    if (rows <= c->pf_rows) return LBK_OK;
    LBK_CUDA(cudaDeviceSynchronize());
    for (void *p : c->pf_allocs) cudaFree(p);
    c->pf_allocs.clear();
    c->pf_rows = 0;
    LBK_TRY(dev_alloc(c->pf_allocs, rows * 4, reinterpret_cast<void **>(&c->pf_tokens)));
    LBK_TRY(dev_alloc(c->pf_allocs, rows * m->cfg.hidden_size * 4, reinterpret_cast<void **>(&c->pf_n)));
    LBK_TRY(dev_alloc(c->pf_allocs, kLogitRows * m->cfg.vocab_size * 4, reinterpret_cast<void **>(&c->pf_logits)));
    LBK_TRY(m->make_prefill_buffers(c, rows));
    c->pf_rows = rows;
    return LBK_OK;
}

// Which rows' logits a pass returns: `n` places (ascending order is not required) or every row.
struct Want {
    const uint32_t *places = nullptr;
    size_t n = 0;
    bool all = false;
};

// `n` (at most the model's prefill_rows) consecutive tokens of sequence `seq` in one pass. `rows[i]` (places
// in this pass) get their logits written to host memory at logits_out[i * vocab]; `next_out` (host) receives
// the greedy token after the last row (sample.rs:17-25). Synchronous.
int run_rows(Model *m, Cache *c, size_t seq, const uint32_t *tokens, size_t n, const std::vector<uint32_t> &rows, float *logits_out,
             int32_t *next_out = nullptr) {
    Ctx *ctx = m->ctx;
    lbk_ctx *h = reinterpret_cast<lbk_ctx *>(ctx);
    cudaStream_t st = ctx->own_stream;
    const size_t H = m->cfg.hidden_size, V = m->cfg.vocab_size;
    LBK_TRY(ensure_prefill_buffers(m, c, n));
    std::vector<int32_t> toks(n);
    for (size_t i = 0; i < n; ++i) toks[i] = static_cast<int32_t>(tokens[i]);
    LBK_CUDA(cudaMemcpyAsync(c->pf_tokens, toks.data(), n * 4, cudaMemcpyHostToDevice, st));
    LBK_CUDA(cudaStreamSynchronize(st));  // `toks` is pageable host memory that goes away
    LBK_TRY(m->enqueue_rows(c, seq, n, st));
    // runs of neighbouring rows go through the head together
    for (size_t i = 0; i < rows.size();) {
        size_t len = 1;
        while (i + len < rows.size() && len < kLogitRows && rows[i + len] == rows[i] + len) ++len;
        LBK_TRY(m->enqueue_head(c->pf_n + rows[i] * H, len, c->pf_logits, st));
        LBK_CUDA(cudaMemcpyAsync(logits_out + i * V, c->pf_logits, len * V * 4, cudaMemcpyDeviceToHost, st));
        LBK_CUDA(cudaStreamSynchronize(st));  // the staging rows are reused by the next run
        i += len;
    }
    if (next_out) {
        LBK_TRY(m->enqueue_head(c->pf_n + (n - 1) * H, 1, c->pf_logits, st));
        LBK_TRY(lbk_argmax(h, c->pf_logits, 1, V, c->pf_tokens, st));  // the token buffer is free again
        LBK_CUDA(cudaMemcpyAsync(next_out, c->pf_tokens, 4, cudaMemcpyDeviceToHost, st));
    }
    const int32_t new_len = static_cast<int32_t>(c->lens[seq] + n);
    LBK_CUDA(cudaStreamSynchronize(st));
    LBK_CUDA(cudaMemcpy(c->pos + seq, &new_len, 4, cudaMemcpyHostToDevice));
    c->lens[seq] += n;
    return LBK_OK;
}

// One decode step of every slot: the family's launches, the greedy token, the positions.
int enqueue_full_step(Model *m, Cache *c, cudaStream_t st) {
    lbk_ctx *h = reinterpret_cast<lbk_ctx *>(m->ctx);
    LBK_TRY(m->enqueue_step(c, st));
    LBK_TRY(lbk_argmax(h, c->logits, c->b, m->cfg.vocab_size, c->next, st));  // sample.rs:17-25
    return lbk_advance_pos_seq(h, c->pos, c->active, c->b, st);
}

// Records the step into a graph on the context's own stream (a few eager steps first: the library's
// scratch buffers must exist before anything is captured; those steps run on a scratch position).
int ensure_graph(Model *m, Cache *c) {
    if (c->step) return LBK_OK;
    Ctx *ctx = m->ctx;
    cudaStream_t st = ctx->own_stream;
    std::vector<int32_t> saved(c->b);
    LBK_CUDA(cudaMemcpy(saved.data(), c->active, c->b * 4, cudaMemcpyDeviceToHost));
    // Eager warm-up with no sequence taking part: positions and recurrent states stay; cache rows written at the present
    // positions are rewritten by the real step.
    LBK_CUDA(cudaMemsetAsync(c->active, 0, c->b * 4, st));
    LBK_TRY(enqueue_full_step(m, c, st));
    LBK_CUDA(cudaMemcpyAsync(c->active, saved.data(), c->b * 4, cudaMemcpyHostToDevice, st));
    LBK_CUDA(cudaStreamSynchronize(st));
    const uint64_t before = ctx->launches;
    LBK_CUDA(cudaStreamBeginCapture(st, cudaStreamCaptureModeThreadLocal));
    const int status = enqueue_full_step(m, c, st);
    cudaGraph_t graph = nullptr;
    const cudaError_t e = cudaStreamEndCapture(st, &graph);
    c->step_launches = ctx->launches - before;
    ctx->launches = before;  // recording is not launching
    if (status != LBK_OK) {
        if (graph) cudaGraphDestroy(graph);
        return status;
    }
    if (e != cudaSuccess) return fail(LBK_ERR_CUDA, "capture of the decode step failed: %s", cudaGetErrorString(e));
    const cudaError_t ei = cudaGraphInstantiate(&c->step, graph, 0);
    cudaGraphDestroy(graph);
    if (ei != cudaSuccess) return fail(LBK_ERR_CUDA, "cudaGraphInstantiate: %s", cudaGetErrorString(ei));
    return LBK_OK;
}

}  // namespace

}  // namespace lbk

using namespace lbk;

namespace {

int load_impl(lbk_ctx *c, const char *directory, int compute, int rank, int world, lbk_model **out) {
    if (!c || !directory || !out) return fail(LBK_ERR_INVALID, "lbk_model_load: null argument");
    *out = nullptr;
    if (world < 1 || rank < 0 || rank >= world) return fail(LBK_ERR_INVALID, "rank %d of %d", rank, world);
    if (compute != LBK_COMPUTE_BF16 && compute != LBK_COMPUTE_F32) return fail(LBK_ERR_INVALID, "unknown compute type %d", compute);
    const double t0 = now_seconds();
    Ctx *ctx = reinterpret_cast<Ctx *>(c);
    LBK_CUDA(cudaSetDevice(ctx->device));
    const std::string dir(directory);
    std::string text;
    if (!read_file(dir + "/config.json", text)) return fail(LBK_ERR_INVALID, "cannot read %s/config.json", directory);
    Json cj;
    if (!parse_json(text, cj) || cj.kind != Json::Obj) return fail(LBK_ERR_INVALID, "%s/config.json is not a JSON object", directory);
    const Json *ja = cj.get("architecture");
    const std::string arch = ja && ja->kind == Json::Str ? ja->str : "";
    const auto it = families().find(arch);
    if (it == families().end()) return fail(LBK_ERR_UNSUPPORTED, "%s/config.json: no model family for architecture \"%s\" in this library", directory, arch.c_str());
    std::unique_ptr<Model> model;
    LBK_TRY(it->second(ctx, dir, cj, compute, rank, world, model));
    LBK_CUDA(cudaStreamSynchronize(ctx->own_stream));
    Model *m = model.get();
    if (m->architecture.empty()) m->architecture = arch.empty() ? "BitNet" : arch;
    m->compute = compute;
    if (!m->prefill_rows) m->prefill_rows = kPrefillChunk;
    m->stats.seconds = now_seconds() - t0;
    m->stats.staging_bytes = 2 * kStageBytes;
    *out = reinterpret_cast<lbk_model *>(model.release());
    return LBK_OK;
}

// Tokens of one sequence, in passes of at most prefill_rows rows; a single token of a one-sequence cache takes
// the recorded decode step.
int forward_impl(Model *m, Cache *c, size_t seq, const uint32_t *tokens, size_t n, const Want &want, float *logits_out) {
    if (c->model != m) return fail(LBK_ERR_INVALID, "the cache belongs to another model");
    if (seq >= c->b) return fail(LBK_ERR_INVALID, "sequence %zu of a cache of %zu", seq, c->b);
    if (n == 0) return LBK_OK;
    if (c->lens[seq] + n > c->cap) return fail(LBK_ERR_INVALID, "%zu tokens do not fit: %zu of %zu positions are used", n, c->lens[seq], c->cap);
    LBK_CUDA(cudaSetDevice(m->ctx->device));
    cudaStream_t st = m->ctx->own_stream;
    const size_t V = m->cfg.vocab_size;
    for (size_t i = 0; i < n; ++i)
        if (tokens[i] >= V) return fail(LBK_ERR_INVALID, "token %u is outside the vocabulary of %zu", tokens[i], V);
    for (size_t i = 0; i < want.n; ++i)
        if (want.places[i] >= n) return fail(LBK_ERR_INVALID, "logits of place %u were asked for, the call has %zu tokens", want.places[i], n);
    std::vector<uint32_t> rows;
    std::vector<size_t> at;   // where in logits_out the pass's rows go
    std::vector<float> part;
    for (size_t i0 = 0; i0 < n;) {
        const size_t take = std::min(m->prefill_rows, n - i0);
        rows.clear();
        at.clear();
        if (want.all) {
            for (size_t i = 0; i < take; ++i) rows.push_back(static_cast<uint32_t>(i));
        } else {
            for (size_t i = 0; i < want.n; ++i)
                if (want.places[i] >= i0 && want.places[i] < i0 + take) {
                    rows.push_back(static_cast<uint32_t>(want.places[i] - i0));
                    at.push_back(i);
                }
        }
        if (take == 1 && c->b == 1) {
            LBK_TRY(ensure_graph(m, c));
            const int32_t tk = static_cast<int32_t>(tokens[i0]);
            LBK_CUDA(cudaMemcpyAsync(c->tokens, &tk, 4, cudaMemcpyHostToDevice, st));
            LBK_CUDA(cudaStreamSynchronize(st));  // `tk` is a stack variable
            LBK_CUDA(cudaGraphLaunch(c->step, st));
            m->ctx->launches += c->step_launches;
            c->lens[0] += 1;
            for (size_t i = 0; i < rows.size(); ++i)
                LBK_CUDA(cudaMemcpyAsync(logits_out + (want.all ? i0 : at[i]) * V, c->logits, V * 4, cudaMemcpyDeviceToHost, st));
            LBK_CUDA(cudaStreamSynchronize(st));
        } else if (want.all) {
            LBK_TRY(run_rows(m, c, seq, tokens + i0, take, rows, logits_out + i0 * V));
        } else {
            // the wanted places of a pass need not be neighbours in the output
            bool straight = true;
            for (size_t i = 1; i < at.size(); ++i) straight = straight && at[i] == at[0] + i;
            if (straight) {
                LBK_TRY(run_rows(m, c, seq, tokens + i0, take, rows, at.empty() ? nullptr : logits_out + at[0] * V));
            } else {
                part.resize(rows.size() * V);
                LBK_TRY(run_rows(m, c, seq, tokens + i0, take, rows, part.data()));
                for (size_t i = 0; i < at.size(); ++i) memcpy(logits_out + at[i] * V, part.data() + i * V, V * 4);
            }
        }
        i0 += take;
    }
    return LBK_OK;
}

}  // namespace

extern "C" {

int lbk_model_free(lbk_model *mp) {
    delete reinterpret_cast<Model *>(mp);
    return LBK_OK;
}

int lbk_model_load(lbk_ctx *c, const char *directory, lbk_model **out) { return load_impl(c, directory, LBK_COMPUTE_BF16, 0, 1, out); }

int lbk_model_load_compute(lbk_ctx *c, const char *directory, int compute, lbk_model **out) { return load_impl(c, directory, compute, 0, 1, out); }

int lbk_model_load_shard(lbk_ctx *c, const char *directory, int rank, int world, lbk_model **out) {
    return load_impl(c, directory, LBK_COMPUTE_BF16, rank, world, out);
}

const char *lbk_model_architecture(const lbk_model *mp) { return mp ? reinterpret_cast<const Model *>(mp)->architecture.c_str() : ""; }

int lbk_model_has_architecture(const char *architecture) { return architecture && families().count(architecture) ? 1 : 0; }

int lbk_model_load_stats(const lbk_model *mp, lbk_load_stats *out) {
    if (!mp || !out) return fail(LBK_ERR_INVALID, "lbk_model_load_stats: null argument");
    *out = reinterpret_cast<const Model *>(mp)->stats;
    return LBK_OK;
}

int lbk_model_get_config(const lbk_model *mp, lbk_model_config *out) {
    if (!mp || !out) return fail(LBK_ERR_INVALID, "lbk_model_get_config: null argument");
    *out = reinterpret_cast<const Model *>(mp)->cfg;
    return LBK_OK;
}

int lbk_kv_cache_free(lbk_kv_cache *cp) {
    delete reinterpret_cast<Cache *>(cp);
    return LBK_OK;
}

int lbk_model_new_cache(lbk_model *mp, size_t batch, size_t capacity, lbk_kv_cache **out) {
    if (!mp || !out) return fail(LBK_ERR_INVALID, "lbk_model_new_cache: null argument");
    *out = nullptr;
    Model *m = reinterpret_cast<Model *>(mp);
    if (batch == 0 || batch > LBK_GEMV_MAX_M) return fail(LBK_ERR_UNSUPPORTED, "a cache serves 1..%d sequences (got %zu)", LBK_GEMV_MAX_M, batch);
    LBK_CUDA(cudaSetDevice(m->ctx->device));
    std::unique_ptr<Cache> cache;
    LBK_TRY(m->make_cache(batch, capacity, cache));
    Cache *c = cache.get();
    c->model = m;
    c->b = batch;
    struct { void **p; size_t bytes; } bufs[] = {
        {reinterpret_cast<void **>(&c->pos), batch * 4}, {reinterpret_cast<void **>(&c->active), batch * 4}, {reinterpret_cast<void **>(&c->tokens), batch * 4},
        {reinterpret_cast<void **>(&c->next), batch * 4}, {reinterpret_cast<void **>(&c->logits), batch * m->cfg.vocab_size * 4}};
    for (auto &bf : bufs) {
        LBK_TRY(dev_alloc(c->device_allocs, bf.bytes, bf.p));
        LBK_CUDA(cudaMemset(*bf.p, 0, bf.bytes));
    }
    c->lens.assign(batch, 0);
    const std::vector<int32_t> ones(batch, 1);
    LBK_CUDA(cudaMemcpy(c->active, ones.data(), batch * 4, cudaMemcpyHostToDevice));
    *out = reinterpret_cast<lbk_kv_cache *>(cache.release());
    return LBK_OK;
}

size_t lbk_kv_cache_len(const lbk_kv_cache *cp) { return cp ? reinterpret_cast<const Cache *>(cp)->lens[0] : 0; }

int lbk_kv_cache_reset(lbk_kv_cache *cp) {
    if (!cp) return fail(LBK_ERR_INVALID, "cache is null");
    Cache *c = reinterpret_cast<Cache *>(cp);
    LBK_CUDA(cudaSetDevice(c->model->ctx->device));
    LBK_CUDA(cudaDeviceSynchronize());
    LBK_CUDA(cudaMemset(c->pos, 0, c->b * 4));
    LBK_CUDA(cudaDeviceSynchronize());  // the context's own stream does not wait for the default one
    c->lens.assign(c->b, 0);
    return LBK_OK;
}

int lbk_model_decode(lbk_model *mp, lbk_kv_cache *cp, const int32_t *tokens_dev, float *logits_dev, int32_t *next_dev, void *stream) {
    if (!mp || !cp || !tokens_dev) return fail(LBK_ERR_INVALID, "lbk_model_decode: null argument");
    Model *m = reinterpret_cast<Model *>(mp);
    Cache *c = reinterpret_cast<Cache *>(cp);
    if (c->model != m) return fail(LBK_ERR_INVALID, "the cache belongs to another model");
    for (size_t l : c->lens)
        if (l >= c->cap) return fail(LBK_ERR_INVALID, "the cache is full (%zu positions)", c->cap);
    LBK_CUDA(cudaSetDevice(m->ctx->device));
    LBK_TRY(ensure_graph(m, c));
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    LBK_CUDA(cudaMemcpyAsync(c->tokens, tokens_dev, c->b * 4, cudaMemcpyDeviceToDevice, st));
    LBK_CUDA(cudaGraphLaunch(c->step, st));
    m->ctx->launches += c->step_launches;
    if (logits_dev) LBK_CUDA(cudaMemcpyAsync(logits_dev, c->logits, c->b * m->cfg.vocab_size * 4, cudaMemcpyDeviceToDevice, st));
    if (next_dev) LBK_CUDA(cudaMemcpyAsync(next_dev, c->next, c->b * 4, cudaMemcpyDeviceToDevice, st));
    for (size_t &l : c->lens) l += 1;
    return LBK_OK;
}

int lbk_model_forward(lbk_model *mp, lbk_kv_cache *cp, const uint32_t *tokens, size_t n, int all_logits, float *logits_out) {
    if (!mp || !cp || (n && !tokens)) return fail(LBK_ERR_INVALID, "lbk_model_forward: null argument");
    Cache *c = reinterpret_cast<Cache *>(cp);
    if (c->b != 1) return fail(LBK_ERR_INVALID, "lbk_model_forward drives one sequence; this cache was made for %zu", c->b);
    if (n == 0) return LBK_OK;
    const uint32_t last = static_cast<uint32_t>(n - 1);
    Want want;
    if (logits_out) {
        want.all = all_logits != 0;
        want.places = &last;
        want.n = want.all ? 0 : 1;
    }
    return forward_impl(reinterpret_cast<Model *>(mp), c, 0, tokens, n, want, logits_out);
}

int lbk_model_forward_rows(lbk_model *mp, lbk_kv_cache *cp, size_t seq, const uint32_t *tokens, size_t n, const uint32_t *want, size_t n_want,
                           float *logits_out) {
    if (!mp || !cp || (n && !tokens) || (n_want && (!want || !logits_out))) return fail(LBK_ERR_INVALID, "lbk_model_forward_rows: null argument");
    Want w;
    w.places = want;
    w.n = n_want;
    return forward_impl(reinterpret_cast<Model *>(mp), reinterpret_cast<Cache *>(cp), seq, tokens, n, w, logits_out);
}

int lbk_kv_cache_reset_seq(lbk_kv_cache *cp, size_t seq) {
    Cache *c = reinterpret_cast<Cache *>(cp);
    if (!c || seq >= c->b) return fail(LBK_ERR_INVALID, "lbk_kv_cache_reset_seq: no such sequence");
    LBK_CUDA(cudaSetDevice(c->model->ctx->device));
    LBK_CUDA(cudaDeviceSynchronize());
    LBK_CUDA(cudaMemset(c->pos + seq, 0, 4));
    LBK_CUDA(cudaDeviceSynchronize());
    c->lens[seq] = 0;
    return LBK_OK;
}

int lbk_model_set_prefill_rows(lbk_model *mp, size_t rows) {
    if (!mp) return fail(LBK_ERR_INVALID, "lbk_model_set_prefill_rows: model is null");
    if (rows < 1 || rows > 8192) return fail(LBK_ERR_INVALID, "rows per prompt pass must be 1..8192 (got %zu)", rows);
    reinterpret_cast<Model *>(mp)->prefill_rows = rows;
    return LBK_OK;
}

size_t lbk_kv_cache_len_seq(const lbk_kv_cache *cp, size_t seq) {
    const Cache *c = reinterpret_cast<const Cache *>(cp);
    return c && seq < c->b ? c->lens[seq] : 0;
}

int lbk_batcher_create(lbk_model *mp, size_t slots, size_t capacity, lbk_batcher **out) {
    if (!mp || !out) return fail(LBK_ERR_INVALID, "lbk_batcher_create: null argument");
    *out = nullptr;
    lbk_kv_cache *cache = nullptr;
    LBK_TRY(lbk_model_new_cache(mp, slots, capacity, &cache));
    Batcher *b = new Batcher();
    b->model = reinterpret_cast<Model *>(mp);
    b->cache = reinterpret_cast<Cache *>(cache);
    b->slot_req.assign(slots, 0);
    *out = reinterpret_cast<lbk_batcher *>(b);
    return LBK_OK;
}

int lbk_batcher_destroy(lbk_batcher *bp) {
    if (!bp) return LBK_OK;
    Batcher *b = reinterpret_cast<Batcher *>(bp);
    lbk_kv_cache_free(reinterpret_cast<lbk_kv_cache *>(b->cache));
    delete b;
    return LBK_OK;
}

int lbk_batcher_submit(lbk_batcher *bp, const uint32_t *prompt, size_t n, size_t max_new_tokens, int32_t eos_token, uint64_t *id_out) {
    if (!bp || !prompt || !id_out) return fail(LBK_ERR_INVALID, "lbk_batcher_submit: null argument");
    Batcher *b = reinterpret_cast<Batcher *>(bp);
    if (n == 0 || max_new_tokens == 0) return fail(LBK_ERR_INVALID, "a request needs a prompt and at least one token to generate");
    if (n > b->cache->cap) return fail(LBK_ERR_INVALID, "a prompt of %zu tokens does not fit %zu positions", n, b->cache->cap);
    const size_t V = b->model->cfg.vocab_size;
    for (size_t i = 0; i < n; ++i)
        if (prompt[i] >= V) return fail(LBK_ERR_INVALID, "token %u is outside the vocabulary of %zu", prompt[i], V);
    Request r;
    r.id = b->next_id++;
    r.prompt.assign(prompt, prompt + n);
    r.max_new = max_new_tokens;
    r.eos = eos_token;
    b->queue.push_back(r.id);
    *id_out = r.id;
    b->reqs.emplace(r.id, std::move(r));
    return LBK_OK;
}

int lbk_batcher_step(lbk_batcher *bp, size_t *pending_out) {
    if (!bp) return fail(LBK_ERR_INVALID, "lbk_batcher_step: null argument");
    Batcher *b = reinterpret_cast<Batcher *>(bp);
    Model *m = b->model;
    Cache *c = b->cache;
    LBK_CUDA(cudaSetDevice(m->ctx->device));
    cudaStream_t st = m->ctx->own_stream;
    const size_t slots = c->b;
    // a sequence is finished by its end token, its budget, or a full cache; its slot goes back at once
    auto finished = [&](const Request &r, size_t slot) {
        return (r.eos >= 0 && static_cast<int32_t>(r.out.back()) == r.eos) || r.out.size() >= r.max_new || c->lens[slot] >= c->cap;
    };
    auto retire = [&](Request &r, size_t slot) -> int {
        r.done = true;
        r.slot = -1;
        b->slot_req[slot] = 0;
        const int32_t zero = 0;  // an idle slot still runs through the step: keep its position inside the cache
        LBK_CUDA(cudaMemcpy(c->pos + slot, &zero, 4, cudaMemcpyHostToDevice));
        c->lens[slot] = 0;
        return LBK_OK;
    };
    // admission: prompts into free slots
    for (size_t slot = 0; slot < slots && !b->queue.empty(); ++slot) {
        if (b->slot_req[slot]) continue;
        Request &r = b->reqs.at(b->queue.front());
        b->queue.pop_front();
        int32_t first = 0;
        for (size_t i0 = 0; i0 < r.prompt.size(); i0 += m->prefill_rows) {
            const size_t rows = std::min(m->prefill_rows, r.prompt.size() - i0);
            const bool last = i0 + rows == r.prompt.size();
            LBK_TRY(run_rows(m, c, slot, r.prompt.data() + i0, rows, {}, nullptr, last ? &first : nullptr));
        }
        r.out.push_back(static_cast<uint32_t>(first));
        r.slot = static_cast<int>(slot);
        b->slot_req[slot] = r.id;
        if (finished(r, slot)) LBK_TRY(retire(r, slot));
    }
    // one decode step for the occupied slots
    std::vector<int32_t> tokens(slots, 0), active(slots, 0), next(slots, 0);
    size_t n_active = 0;
    for (size_t slot = 0; slot < slots; ++slot)
        if (b->slot_req[slot]) {
            tokens[slot] = static_cast<int32_t>(b->reqs.at(b->slot_req[slot]).out.back());
            active[slot] = 1;
            ++n_active;
        }
    if (n_active) {
        LBK_TRY(ensure_graph(m, c));
        LBK_CUDA(cudaMemcpyAsync(c->tokens, tokens.data(), slots * 4, cudaMemcpyHostToDevice, st));
        LBK_CUDA(cudaMemcpyAsync(c->active, active.data(), slots * 4, cudaMemcpyHostToDevice, st));
        LBK_CUDA(cudaStreamSynchronize(st));  // the host vectors are pageable
        LBK_CUDA(cudaGraphLaunch(c->step, st));
        m->ctx->launches += c->step_launches;
        LBK_CUDA(cudaMemcpyAsync(next.data(), c->next, slots * 4, cudaMemcpyDeviceToHost, st));
        LBK_CUDA(cudaStreamSynchronize(st));
        for (size_t slot = 0; slot < slots; ++slot) {
            if (!b->slot_req[slot]) continue;
            Request &r = b->reqs.at(b->slot_req[slot]);
            c->lens[slot] += 1;
            r.out.push_back(static_cast<uint32_t>(next[slot]));
            if (finished(r, slot)) LBK_TRY(retire(r, slot));
        }
    }
    if (pending_out) {
        size_t occupied = 0;
        for (uint64_t id : b->slot_req) occupied += id != 0;
        *pending_out = occupied + b->queue.size();
    }
    return LBK_OK;
}

int lbk_batcher_poll(lbk_batcher *bp, uint64_t id, uint32_t *tokens_out, size_t capacity, size_t *n_out, int *done_out) {
    if (!bp || !n_out) return fail(LBK_ERR_INVALID, "lbk_batcher_poll: null argument");
    Batcher *b = reinterpret_cast<Batcher *>(bp);
    auto it = b->reqs.find(id);
    if (it == b->reqs.end()) return fail(LBK_ERR_INVALID, "no request %llu", static_cast<unsigned long long>(id));
    const Request &r = it->second;
    *n_out = r.out.size();
    if (tokens_out)
        for (size_t i = 0; i < r.out.size() && i < capacity; ++i) tokens_out[i] = r.out[i];
    if (done_out) *done_out = r.done ? 1 : 0;
    return LBK_OK;
}

int lbk_batcher_forget(lbk_batcher *bp, uint64_t id) {
    if (!bp) return fail(LBK_ERR_INVALID, "lbk_batcher_forget: null argument");
    Batcher *b = reinterpret_cast<Batcher *>(bp);
    auto it = b->reqs.find(id);
    if (it == b->reqs.end()) return fail(LBK_ERR_INVALID, "no request %llu", static_cast<unsigned long long>(id));
    if (!it->second.done) return fail(LBK_ERR_INVALID, "request %llu is still running", static_cast<unsigned long long>(id));
    b->reqs.erase(it);
    return LBK_OK;
}

}  // extern "C"
