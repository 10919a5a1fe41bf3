// What the model runtime (lbk_model.cu) and the model families (lbk_bitnet.cu, lbk_pefolix.cu, lbk_dugulorn.cu) share:
// the JSON reader, the safetensors file and its staged copies to the device, and the two base classes. A family
// derives from Model and Cache, registers a loader under the architecture name its config.json carries, and
// supplies the launches of a decode step and of a prompt pass; positions, slots, graphs, logits rows, greedy
// tokens and the batcher are the runtime's.
#pragma once

#include <fcntl.h>
#include <sys/stat.h>
#include <time.h>
#include <unistd.h>

#include <algorithm>
#include <cmath>
#include <cstdio>
#include <cstdlib>
#include <cstring>
#include <map>
#include <memory>
#include <string>
#include <vector>

#include "lbk_dense.cuh"
#include "lbk_internal.cuh"

namespace lbk {

// ---- a small JSON reader (objects, arrays, strings, numbers, true/false/null) -----------------
struct Json {
    enum Kind { Null, Bool, Num, Str, Arr, Obj } kind = Null;
    bool b = false;
    double num = 0.0;
    std::string str;
    std::vector<Json> arr;
    std::vector<std::pair<std::string, Json>> obj;
    const Json *get(const char *key) const {
        for (const auto &kv : obj)
            if (kv.first == key) return &kv.second;
        return nullptr;
    }
};

struct JsonParser {
    const char *p, *end;
    bool ok = true;
    void ws() {
        while (p < end && (*p == ' ' || *p == '\n' || *p == '\t' || *p == '\r')) ++p;
    }
    bool lit(const char *s) {
        const size_t n = strlen(s);
        if (static_cast<size_t>(end - p) >= n && memcmp(p, s, n) == 0) {
            p += n;
            return true;
        }
        return false;
    }
    std::string string() {
        std::string out;
        if (p >= end || *p != '"') {
            ok = false;
            return out;
        }
        ++p;
        while (p < end && *p != '"') {
            if (*p == '\\' && p + 1 < end) {
                ++p;
                switch (*p) {
                    case 'n': out += '\n'; break;
                    case 't': out += '\t'; break;
                    case 'r': out += '\r'; break;
                    case 'b': out += '\b'; break;
                    case 'f': out += '\f'; break;
                    case 'u':  // keep the escape as text: tensor names and the fields read here are ASCII
                        out += "\\u";
                        break;
                    default: out += *p;
                }
                ++p;
            } else {
                out += *p++;
            }
        }
        if (p >= end) ok = false;
        else ++p;
        return out;
    }
    Json value(int depth = 0) {
        Json j;
        ws();
        if (p >= end || depth > 64) {
            ok = false;
            return j;
        }
        if (*p == '{') {
            j.kind = Json::Obj;
            ++p;
            ws();
            if (p < end && *p == '}') {
                ++p;
                return j;
            }
            while (ok) {
                ws();
                std::string key = string();
                ws();
                if (!ok || p >= end || *p != ':') {
                    ok = false;
                    break;
                }
                ++p;
                j.obj.emplace_back(std::move(key), value(depth + 1));
                ws();
                if (p < end && *p == ',') {
                    ++p;
                    continue;
                }
                if (p < end && *p == '}') {
                    ++p;
                    break;
                }
                ok = false;
            }
        } else if (*p == '[') {
            j.kind = Json::Arr;
            ++p;
            ws();
            if (p < end && *p == ']') {
                ++p;
                return j;
            }
            while (ok) {
                j.arr.push_back(value(depth + 1));
                ws();
                if (p < end && *p == ',') {
                    ++p;
                    continue;
                }
                if (p < end && *p == ']') {
                    ++p;
                    break;
                }
                ok = false;
            }
        } else if (*p == '"') {
            j.kind = Json::Str;
            j.str = string();
        } else if (lit("true")) {
            j.kind = Json::Bool;
            j.b = true;
        } else if (lit("false")) {
            j.kind = Json::Bool;
        } else if (lit("null")) {
            j.kind = Json::Null;
        } else {
            char *e = nullptr;
            j.kind = Json::Num;
            j.num = strtod(p, &e);
            if (e == p || e > end) ok = false;
            else p = e;
        }
        return j;
    }
};

inline bool parse_json(const std::string &text, Json &out) {
    JsonParser ps{text.data(), text.data() + text.size()};
    out = ps.value();
    ps.ws();
    return ps.ok && ps.p == ps.end;
}

inline bool read_file(const std::string &path, std::string &out) {
    FILE *f = fopen(path.c_str(), "rb");
    if (!f) return false;
    std::string data;
    char buf[1 << 16];
    size_t n;
    while ((n = fread(buf, 1, sizeof(buf), f)) > 0) data.append(buf, n);
    fclose(f);
    out.swap(data);
    return true;
}

struct TensorEntry {
    std::string dtype;
    std::vector<size_t> shape;
    size_t begin = 0, end = 0;  // byte range inside the data section
};

// ---- a safetensors file -> the device: pread into one of two pinned buffers, one copy per piece ----
constexpr size_t kStageBytes = 32u << 20;

struct Stager {
    int fd = -1;
    size_t file_size = 0, data0 = 0;
    cudaStream_t st = nullptr;
    unsigned char *buf[2] = {nullptr, nullptr};
    cudaEvent_t done[2] = {nullptr, nullptr};
    bool busy[2] = {false, false};
    int next = 0;
    size_t bytes_read = 0, bytes_to_device = 0;
    ~Stager() {
        for (int i = 0; i < 2; ++i) {
            if (busy[i]) cudaEventSynchronize(done[i]);
            if (done[i]) cudaEventDestroy(done[i]);
            if (buf[i]) cudaFreeHost(buf[i]);
        }
        if (fd >= 0) close(fd);
    }
    int init(cudaStream_t stream) {
        st = stream;
        for (int i = 0; i < 2; ++i) {
            cudaError_t e = cudaMallocHost(reinterpret_cast<void **>(&buf[i]), kStageBytes);
            if (e != cudaSuccess) return fail(LBK_ERR_NOMEM, "pinned staging buffer: %s", cudaGetErrorString(e));
            LBK_CUDA(cudaEventCreateWithFlags(&done[i], cudaEventDisableTiming));
        }
        return LBK_OK;
    }
    int acquire(int *slot) {
        const int s = next;
        next ^= 1;
        if (busy[s]) {
            LBK_CUDA(cudaEventSynchronize(done[s]));
            busy[s] = false;
        }
        *slot = s;
        return LBK_OK;
    }
    int fill(int s, size_t file_off, size_t n, const char *what) {
        if (file_off + n > file_size) return fail(LBK_ERR_INVALID, "the file is truncated: %s needs bytes up to %zu, the file has %zu", what, file_off + n, file_size);
        size_t got = 0;
        while (got < n) {
            const ssize_t r = pread(fd, buf[s] + got, n - got, static_cast<off_t>(file_off + got));
            if (r <= 0) return fail(LBK_ERR_INVALID, "cannot read %s (%zu of %zu bytes)", what, got, n);
            got += static_cast<size_t>(r);
        }
        bytes_read += n;
        return LBK_OK;
    }
    int release(int s) {
        LBK_CUDA(cudaEventRecord(done[s], st));
        busy[s] = true;
        return LBK_OK;
    }
    // `n` contiguous bytes at data offset `off` -> dst
    int copy_linear(size_t off, size_t n, void *dst, const char *what) {
        for (size_t o = 0; o < n; o += kStageBytes) {
            const size_t len = n - o < kStageBytes ? n - o : kStageBytes;
            int s;
            LBK_TRY(acquire(&s));
            LBK_TRY(fill(s, data0 + off + o, len, what));
            LBK_CUDA(cudaMemcpyAsync(static_cast<char *>(dst) + o, buf[s], len, cudaMemcpyHostToDevice, st));
            bytes_to_device += len;
            LBK_TRY(release(s));
        }
        return LBK_OK;
    }
    // `rows` rows of `width` contiguous bytes at data offset `off` -> dst, rows `pitch` bytes apart there
    int copy_rows(size_t off, size_t rows, size_t width, void *dst, size_t pitch, const char *what) {
        const size_t rows_per = width ? kStageBytes / width : 0;
        if (rows_per == 0) return fail(LBK_ERR_UNSUPPORTED, "%s: a row of %zu bytes does not fit the staging buffer", what, width);
        for (size_t r = 0; r < rows; r += rows_per) {
            const size_t nr = rows - r < rows_per ? rows - r : rows_per;
            int s;
            LBK_TRY(acquire(&s));
            LBK_TRY(fill(s, data0 + off + r * width, nr * width, what));
            LBK_CUDA(cudaMemcpy2DAsync(static_cast<char *>(dst) + r * pitch, pitch, buf[s], width, width, nr, cudaMemcpyHostToDevice, st));
            bytes_to_device += nr * width;
            LBK_TRY(release(s));
        }
        return LBK_OK;
    }
    // bytes [c0, c0 + width) of each of `rows` rows of pitch `pitch` starting at data offset `off` -> dst (pitch = width)
    int copy_columns(size_t off, size_t rows, size_t pitch, size_t c0, size_t width, void *dst, const char *what) {
        const size_t rows_per = kStageBytes / pitch;
        if (rows_per == 0) return fail(LBK_ERR_UNSUPPORTED, "%s: a row of %zu bytes does not fit the staging buffer", what, pitch);
        for (size_t r = 0; r < rows; r += rows_per) {
            const size_t nr = rows - r < rows_per ? rows - r : rows_per;
            int s;
            LBK_TRY(acquire(&s));
            LBK_TRY(fill(s, data0 + off + r * pitch, nr * pitch, what));
            LBK_CUDA(cudaMemcpy2DAsync(static_cast<char *>(dst) + r * width, width, buf[s] + c0, pitch, width, nr, cudaMemcpyHostToDevice, st));
            bytes_to_device += nr * width;
            LBK_TRY(release(s));
        }
        return LBK_OK;
    }
};

inline double now_seconds() {
    timespec ts;
    clock_gettime(CLOCK_MONOTONIC, &ts);
    return static_cast<double>(ts.tv_sec) + 1e-9 * static_cast<double>(ts.tv_nsec);
}

// u64 header length, JSON header, data. `format` (may be empty) receives __metadata__.format.
struct TensorFile {
    std::string path;
    Stager sg;
    std::map<std::string, TensorEntry> entries;
    std::string format;
    int open_file(const std::string &file, cudaStream_t stream);
    // the entry `name`, checked: dtype, number of elements, bytes inside the file
    int find(const std::string &name, const char *dtype, size_t elems, size_t elem_bytes, const TensorEntry **out) const;
};

inline int dev_alloc(std::vector<void *> &owner, size_t bytes, void **out) {
    void *p = nullptr;
    cudaError_t e = cudaMalloc(&p, bytes ? bytes : 16);
    if (e != cudaSuccess) return fail(LBK_ERR_NOMEM, "cudaMalloc(%zu) failed: %s", bytes, cudaGetErrorString(e));
    owner.push_back(p);
    *out = p;
    return LBK_OK;
}

inline size_t json_size(const Json *j, bool &ok) {
    if (!j || j->kind != Json::Num || j->num < 0) {
        ok = false;
        return 0;
    }
    return static_cast<size_t>(j->num);
}

// ---- weights of a family from its tensor file (bf16 tensors) -----------------------------------------
struct WeightLoader {
    Ctx *ctx;
    std::vector<void *> &owner;  // who frees the device memory
    TensorFile &tf;

    // rows and columns of a matrix
    int shape(const std::string &name, size_t *rows, size_t *cols) const;
    // n values as f32 on the host
    int read(const std::string &name, size_t n, std::vector<float> &out);
    // a vector as f32, `add` added to every value
    int vec(const std::string &name, size_t n, float **out, float add = 0.0f);
    // numbers that are not in the file
    int floats(const std::vector<float> &v, float **out);
    // matrices of the same width, one under the other; an empty name stands for that many rows of zeros
    int stack(const std::vector<std::string> &names, const std::vector<size_t> &rows, size_t cols, DenseWeight *out);
    // a table [rows][cols], rows back to back
    int table(const std::string &name, size_t rows, size_t cols, uint16_t **out);
};
// a whole number of at least 1
bool json_positive(const Json *j, size_t *out);

// ---- the base classes ---------------------------------------------------------------------------
struct Model;

// The sequences ("slots") a model serves together. The family's class adds its K/V rows and work buffers.
struct Cache {
    Model *model = nullptr;
    size_t b = 0, cap = 0;
    int32_t *pos = nullptr;               // [b] length of every sequence, on the device
    int32_t *active = nullptr;            // [b] 1: the sequence takes part in the step (its position advances)
    std::vector<size_t> lens;             // the lengths again, on the host
    int32_t *tokens = nullptr, *next = nullptr;
    float *logits = nullptr;              // [b][vocab] of the last decode step
    cudaGraphExec_t step = nullptr;       // the recorded decode step
    uint64_t step_launches = 0;           // kernels in it
    std::vector<void *> device_allocs;
    // prompt path, sized for pf_rows rows; pf_n: the final norm of every row of the pass, f32 [rows][hidden]
    size_t pf_rows = 0;
    std::vector<void *> pf_allocs;
    int32_t *pf_tokens = nullptr;
    float *pf_n = nullptr, *pf_logits = nullptr;
    virtual ~Cache();
};

struct Model {
    Ctx *ctx = nullptr;
    lbk_model_config cfg{};
    std::string architecture;
    size_t prefill_rows = 0;    // prompt rows per pass (lbk_model_set_prefill_rows)
    std::vector<void *> device_allocs;
    int rank = 0, world = 1;    // tensor-parallel shard this model holds (lbk_model_load_shard)
    int compute = LBK_COMPUTE_BF16;
    lbk_load_stats stats{};
    virtual ~Model();
    // a cache of the family's class with its own buffers; the runtime fills in the common part
    virtual int make_cache(size_t batch, size_t capacity, std::unique_ptr<Cache> &out) = 0;
    // prompt work buffers for `rows` rows (the old ones are gone): everything but pf_tokens, pf_n, pf_logits
    virtual int make_prefill_buffers(Cache *c, size_t rows) = 0;
    // one token per sequence: c->tokens at c->pos -> c->logits (positions not advanced)
    virtual int enqueue_step(Cache *c, cudaStream_t st) = 0;
    // c->pf_tokens[0 .. n) of sequence `seq` at its position -> c->pf_n (position not advanced)
    virtual int enqueue_rows(Cache *c, size_t seq, size_t n, cudaStream_t st) = 0;
    // rows of the final norm -> logits
    virtual int enqueue_head(const float *rows, size_t n, float *logits, cudaStream_t st) = 0;
};

// A family's loader: `config` is the parsed config.json of `dir`.
using LoadFn = int (*)(Ctx *ctx, const std::string &dir, const Json &config, int compute, int rank, int world, std::unique_ptr<Model> &out);
struct FamilyRegistrar {
    // `architecture`: the value of config.json's "architecture", or "" for files that do not have the key
    FamilyRegistrar(const char *architecture, LoadFn load);
};

constexpr size_t kPrefillChunk = 4096;  // prompt rows per pass unless lbk_model_set_prefill_rows says otherwise

}  // namespace lbk
