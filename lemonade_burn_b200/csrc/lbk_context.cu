// The library's base: error messages, tensor maps, the context with its scratch memory. Everything here is
// independent of which kernels are linked in: a kernel file registers what it has to set up per context
// (InitHook), so a library can hold a subset of them.
#include <cstdlib>
#include <cstring>
#include <new>
#include <vector>

#include "lbk_internal.cuh"

namespace lbk {

// ---- errors --------------------------------------------------------------------------
static thread_local char g_err[512] = "";

void set_error(const char *fmt, ...) {
    va_list ap;
    va_start(ap, fmt);
    vsnprintf(g_err, sizeof(g_err), fmt, ap);
    va_end(ap);
}

int fail(int status, const char *fmt, ...) {
    va_list ap;
    va_start(ap, fmt);
    vsnprintf(g_err, sizeof(g_err), fmt, ap);
    va_end(ap);
    return status;
}

// ---- tensor maps ---------------------------------------------------------------------
using EncodeTiledFn = CUresult (*)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *,
                                   const cuuint64_t *, const cuuint64_t *, const cuuint32_t *,
                                   const cuuint32_t *, CUtensorMapInterleave, CUtensorMapSwizzle,
                                   CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

static EncodeTiledFn encode_fn() {
    static EncodeTiledFn fn = nullptr;
    if (!fn) {
        void *p = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) == cudaSuccess &&
            q == cudaDriverEntryPointSuccess)
            fn = reinterpret_cast<EncodeTiledFn>(p);
    }
    return fn;
}

static int encode_2d_u8(CUtensorMap *map, const void *base, uint64_t inner, uint64_t outer,
                        uint64_t pitch, uint32_t box_inner, uint32_t box_outer,
                        CUtensorMapSwizzle swz) {
    EncodeTiledFn fn = encode_fn();
    if (!fn) return fail(LBK_ERR_CUDA, "cuTensorMapEncodeTiled is not available from this driver");
    cuuint64_t dims[2] = {inner, outer};
    cuuint64_t strides[1] = {pitch};
    cuuint32_t box[2] = {box_inner, box_outer};
    cuuint32_t estr[2] = {1, 1};
    CUresult r = fn(map, CU_TENSOR_MAP_DATA_TYPE_UINT8, 2, const_cast<void *>(base), dims, strides, box,
                    estr, CU_TENSOR_MAP_INTERLEAVE_NONE, swz, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                    CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) return fail(LBK_ERR_CUDA, "cuTensorMapEncodeTiled failed with CUresult %d", (int)r);
    return LBK_OK;
}

int encode_bytes_map(CUtensorMap *map, const void *base, size_t inner, size_t outer, size_t pitch, int box_inner, int box_outer) {
    return encode_2d_u8(map, base, inner, outer, pitch, static_cast<uint32_t>(box_inner), static_cast<uint32_t>(box_outer), CU_TENSOR_MAP_SWIZZLE_128B);
}

// Grow-only scratch. A block that has been handed out is never freed before the context is
// destroyed: a CUDA graph recorded by a caller (a decode step captured at 5..8 sequences, whose
// projections take the quantise + GEMM path) has this address baked in, and a later, larger request
// must not turn it into a dangling pointer. A larger request gets a new block; the old ones stay
// (each at least 1.25x its predecessor, so together they hold less than five times the largest).
int ctx_scratch(Ctx *ctx, size_t bytes, void **out) {
    if (bytes > ctx->scratch_bytes) {
        const size_t want = bytes + (bytes >> 2) + 4096;
        void *fresh = nullptr;
        cudaError_t e = cudaMalloc(&fresh, want);
        if (e != cudaSuccess) return fail(LBK_ERR_NOMEM, "cudaMalloc(%zu) failed: %s", want, cudaGetErrorString(e));
        if (ctx->scratch) ctx->retired_scratch.push_back(ctx->scratch);
        ctx->scratch = fresh;
        ctx->scratch_bytes = want;
    }
    *out = ctx->scratch;
    return LBK_OK;
}

// What a non-zero error word means. Code 7 is written by the decoder-step kernels when a position
// read from device memory lies outside the cache; every other code marks a bounded wait that ran out.
int device_error_status(int word) {
    if (word == 7)
        return fail(LBK_ERR_INVALID, "a decode position was outside its cache (position < 0 or >= capacity); the kernels of that step "
                                     "refused to run and its results are invalid");
    return fail(LBK_ERR_TIMEOUT, "a bounded device-side wait gave up (code %d); results of that launch are invalid", word);
}

namespace {
std::vector<InitFn> &init_functions() {
    static std::vector<InitFn> v;
    return v;
}
}  // namespace

InitHook::InitHook(InitFn fn) { init_functions().push_back(fn); }

}  // namespace lbk

using namespace lbk;

static Ctx *C_(lbk_ctx *c) { return reinterpret_cast<Ctx *>(c); }

extern "C" {

const char *lbk_last_error(void) { return g_err; }
int lbk_abi_version(void) { return 1; }

int lbk_init(int device, lbk_ctx **out) {
    if (!out) return fail(LBK_ERR_INVALID, "lbk_init: out is null");
    *out = nullptr;
    int count = 0;
    cudaError_t e = cudaGetDeviceCount(&count);
    if (e != cudaSuccess || count == 0)
        return fail(LBK_ERR_CUDA, "no CUDA device: %s", e == cudaSuccess ? "device count is 0" : cudaGetErrorString(e));
    if (device < 0 || device >= count) return fail(LBK_ERR_INVALID, "device %d out of range (0..%d)", device, count - 1);
    cudaDeviceProp prop;
    LBK_CUDA(cudaGetDeviceProperties(&prop, device));
    if (prop.major != 10)
        return fail(LBK_ERR_UNSUPPORTED, "device %d is sm_%d%d; this library is built for sm_100a only", device, prop.major, prop.minor);
    LBK_CUDA(cudaSetDevice(device));
    Ctx *ctx = new (std::nothrow) Ctx();
    if (!ctx) return fail(LBK_ERR_NOMEM, "out of host memory");
    ctx->device = device;
    ctx->sm_count = prop.multiProcessorCount;
    ctx->smem_optin = prop.sharedMemPerBlockOptin;
    if (cudaMalloc(&ctx->small_scratch, kSmallScratchBytes) != cudaSuccess || cudaMalloc(&ctx->err_word, sizeof(int)) != cudaSuccess || cudaMemset(ctx->err_word, 0, sizeof(int)) != cudaSuccess ||
        cudaStreamCreateWithFlags(&ctx->own_stream, cudaStreamNonBlocking) != cudaSuccess) {
        delete ctx;
        return fail(LBK_ERR_CUDA, "context setup failed: %s", cudaGetErrorString(cudaGetLastError()));
    }
    for (InitFn fn : init_functions()) {
        const int s = fn(ctx);
        if (s != LBK_OK) {
            lbk_destroy(reinterpret_cast<lbk_ctx *>(ctx));
            return s;
        }
    }
    *out = reinterpret_cast<lbk_ctx *>(ctx);
    return LBK_OK;
}

int lbk_destroy(lbk_ctx *c) {
    if (!c) return LBK_OK;
    Ctx *ctx = C_(c);
    cudaSetDevice(ctx->device);
    cudaDeviceSynchronize();
    if (ctx->scratch) cudaFree(ctx->scratch);
    for (void *p : ctx->retired_scratch) cudaFree(p);
    if (ctx->err_word) cudaFree(ctx->err_word);
    if (ctx->small_scratch) cudaFree(ctx->small_scratch);
    if (ctx->gemm_acc) cudaFree(ctx->gemm_acc);
    if (ctx->bf16_x) cudaFree(ctx->bf16_x);
    if (ctx->few_parts) cudaFree(ctx->few_parts);
    if (ctx->own_stream) cudaStreamDestroy(ctx->own_stream);
    delete ctx;
    return LBK_OK;
}

int lbk_check_device_error(lbk_ctx *c) {
    if (!c) return fail(LBK_ERR_INVALID, "context is null");
    Ctx *ctx = C_(c);
    LBK_CUDA(cudaSetDevice(ctx->device));
    LBK_CUDA(cudaDeviceSynchronize());
    int word = 0;
    LBK_CUDA(cudaMemcpy(&word, ctx->err_word, sizeof(int), cudaMemcpyDeviceToHost));
    if (word != 0) {
        LBK_CUDA(cudaMemset(ctx->err_word, 0, sizeof(int)));
        // a launch that gave up may have left partial sums in the split-K buffer, which is zero at rest
        if (ctx->gemm_acc) LBK_CUDA(cudaMemset(ctx->gemm_acc, 0, kGemmAccBytes));
        return device_error_status(word);
    }
    return LBK_OK;
}

uint64_t lbk_launch_count(const lbk_ctx *c) { return c ? reinterpret_cast<const Ctx *>(c)->launches : 0; }

}  // extern "C"
