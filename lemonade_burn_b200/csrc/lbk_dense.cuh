// Shared by the dense bf16-weight kernels (projections, experts) and the families that call them.
#pragma once

#include "lbk_internal.cuh"

namespace lbk {

// A bf16 matrix [rows][pitch] on the device; columns cols .. pitch-1 hold zeros. pitch is a multiple of 64.
struct DenseWeight {
    const uint16_t *w = nullptr;
    size_t rows = 0, cols = 0, pitch = 0;
};
inline size_t dense_pitch(size_t cols) { return (cols + 63) / 64 * 64; }
inline size_t pad16(size_t v) { return (v + 15) / 16 * 16; }

constexpr int kActNone = 0, kActRelu2 = 1, kActSilu = 2;
constexpr int kEpiF32 = 0;   // f32 rows: out[t * ld + r]
constexpr int kEpiElem = 1;  // act(v) in the compute type; rows from f32_from on as f32 into out2[t * ld2 + r - f32_from]
constexpr int kEpiQkv = 2;   // rows of a stacked [q; k; v] projection: q to its buffer, k and v into the cache at the token's position

// What happens to the value of (token t, output row r).
struct DenseEpi {
    int kind = kEpiF32, act = kActNone;
    int act_rows = 1 << 30;      // kEpiElem: output rows below this one get the activation
    const float *bias = nullptr; // [out_rows], added first (not with gated)
    void *out = nullptr;
    long ld = 0;
    int f32_from = 1 << 30;
    float *out2 = nullptr;
    long ld2 = 0;
    // kEpiQkv: q [t][heads][dimp] in `out` (ld = heads * dimp); caches [seq][kv_heads][cap][dimp / vdimp]
    int q_rows = 0, k_rows = 0, dim = 1, dimp = 1, vdim = 1, vdimp = 1, kv_heads = 1, cap = 0;
    int q_split = 1 << 30, q_gap = 0;  // dimensions of a q head from q_split on go q_gap places further
    void *kc = nullptr, *vc = nullptr;
    const int *pos = nullptr;  // decode: one position per token (= sequence); rows: pos[0] is the first token's
    int rows_of_seq = -1;      // >= 0: the tokens are consecutive positions of this sequence; -1: token t is sequence t
    int *err_word = nullptr;
};

// The norms in front of a projection, done inside the few-row kernel (kPreNone: the input rows are ready).
constexpr int kPreNone = 0;
constexpr int kPreNorm = 1;     // n = norm(x) * w
constexpr int kPreAddNorm = 2;  // s = x + norm(y) * w_post (written to xout), n = norm(s) * w (w null: n = s)
struct DensePre {
    int mode = kPreNone;
    bool rms = false;           // the norms divide by the root mean square, without taking the mean off
    const float *x = nullptr, *y = nullptr, *w_post = nullptr, *w = nullptr;
    float *xout = nullptr;
    void *nout = nullptr;  // optional: the normalised rows in the compute type, pitch ldn
    long ldn = 0;
    float eps = 0.0f;
};
bool dense_pre_supported(size_t m, size_t cols);

// x: rows of the compute type, pitch ldx elements (>= w.pitch rounded up to 64, zeros or numbers past cols).
// gated: w holds [gate; up] (rows/2 each, up at row up_row) and the value is gelu_tanh(gate) * up.
struct DenseCall {
    int compute = LBK_COMPUTE_BF16;
    const void *x = nullptr;
    long ldx = 0;
    size_t m = 0;
    DenseWeight w;
    bool gated = false;
    size_t up_row = 0, out_rows = 0;
    DenseEpi epi;
    DensePre pre;
    // experts: w holds `experts` matrices stacked group_rows apart; tokens sorted by expert, expert e's are
    // x rows offs[e] .. offs[e+1]-1 (device) and so are its output rows
    int experts = 0;
    size_t group_rows = 0;
    const int *offs = nullptr;
    const int *gather = nullptr;  // f32 only: x row of sorted row p (null: row p)
};
int launch_dense(Ctx *ctx, const DenseCall &c, cudaStream_t st);

// Which keys a query sees and how distance enters its scores.
struct AttnMask {
    int size = 1 << 30;     // sliding window: distance < size ...
    int keep_first = 0;     // ... or key position < keep_first
    bool alibi = true;      // scores - 2^(-8 (h + 1) / heads) * distance
};
struct AttnCall {
    int compute = LBK_COMPUTE_BF16;
    const void *q = nullptr;  // [rows][heads][dimp] of the compute type
    const void *kc = nullptr, *vc = nullptr;
    const int *pos = nullptr;
    size_t n = 0;             // rows
    int rows_of_seq = -1;     // as in DenseEpi
    size_t heads = 0, kv_heads = 0, dim = 0, dimp = 0, vdim = 0, vdimp = 0, cap = 0;
    float scale = 1.0f;
    AttnMask mask;
    float *scratch = nullptr; // decode: attn_window_scratch floats
    void *out = nullptr;      // [rows][heads * vdim] of the compute type, pitch ldo
    long ldo = 0;
    // prompt rows on tcgen05 only: a second part of every key, the same for all heads (rows of k2_pitch values by
    // position); a query head is [dimp | dim2p] then. And a gate per row and head: the output times sigmoid(gate).
    const void *k2 = nullptr;
    size_t dim2p = 0, k2_pitch = 0, k2_rows = 0;
    const float *gate = nullptr;
    long ldg = 0;
};
size_t attn_window_scratch(size_t b, size_t heads, size_t vdimp, size_t splits);
size_t attn_window_splits(size_t cap, const AttnMask &mask);
int launch_attn_window(Ctx *ctx, const AttnCall &c, cudaStream_t st);
// the tcgen05 form of it for prompt rows (lbk_attn_tc.cu); bf16, dim and vdim at most 128 (with k2: three pieces of 64)
int launch_attn_window_tc(Ctx *ctx, const AttnCall &c, cudaStream_t st);

// ---- norms (lbk_layernorm.cu) -------------------------------------------------------------------
// x += norm(y) * w_post (y null: x as it is); then n = norm(x) * w to out_f (f32, pitch n; may be x itself) and / or
// out_e (compute type, pitch lde). w null: n is the sum itself. norm: layer norm, or with `rms` the RMS norm. The sublayer's rows are y, or with `moe` the expert outputs.
struct MoeOut {
    const uint16_t *rows16 = nullptr;  // expert outputs by sorted row, bf16 or f32, pitch ld
    const float *rows32 = nullptr;
    const int *place = nullptr;        // [t][top] sorted row of each chosen expert
    const float *weight = nullptr;     // [t][top]
    int top = 0;
    const float *shared = nullptr;     // [t][n] f32 or null
    const float *gate = nullptr;       // gate logit of token t at gate[t * ldg]
    long ldg = 0, ld = 0;
};
struct NormCall {
    int compute = LBK_COMPUTE_BF16;
    bool rms = false;
    float *x = nullptr;
    const float *y = nullptr, *w_post = nullptr, *w = nullptr;
    const MoeOut *moe = nullptr;
    size_t rows = 0, n = 0;
    float eps = 0.0f;
    float *out_f = nullptr;
    void *out_e = nullptr;
    long lde = 0;
};
int launch_sandwich_norm(Ctx *ctx, const NormCall &c, cudaStream_t st);

// ---- mixture of experts (lbk_moe.cu) ------------------------------------------------------------
// Scratch of one routed pass, all on the device.
struct MoeRoute {
    int *ids = nullptr, *place = nullptr;      // [n][top]
    float *weight = nullptr;                   // [n][top]
    int *counts = nullptr, *offs = nullptr, *cursor = nullptr;  // [experts + 1]
    int *token = nullptr;                      // [n * top] token of sorted row p
};
size_t moe_route_ints(size_t n, size_t experts, size_t top);
void moe_route_carve(MoeRoute &r, int *base, size_t n, size_t experts, size_t top);
// softmax over the router logits z [n][ldz], the `top` largest, the sorted order; x rows (bf16, pitch ldx) copied
// to xs in that order when xs is given
int launch_moe_route(Ctx *ctx, const float *z, long ldz, size_t n, size_t experts, size_t top, const MoeRoute &r, const void *x, long ldx, void *xs,
                     cudaStream_t st);
// Few tokens (at most LBK_GEMV_MAX_M), bf16: chosen experts' up projections with the routing weight folded in,
// then all down projections (shared expert included) into y f32 [m][out_rows].
struct MoeFewCall {
    const uint16_t *n = nullptr;   // [m][ldn] bf16 input rows
    long ldn = 0;
    size_t m = 0;
    const float *z = nullptr;      // router logits [m][ldz], the gate logit at column experts (when shared)
    long ldz = 0;
    int experts = 0, top = 0;
    DenseWeight up, down;          // stacked: experts * ff rows; experts * width rows
    size_t ff = 0, width = 0;
    uint16_t *h = nullptr;         // [m * top][down.pitch]
    const uint16_t *hs = nullptr;  // shared expert's activations [m][shared_down.pitch] or null
    DenseWeight shared_down;
    int *act = nullptr;            // moe_few_act_ints: the list of chosen experts, up kernel -> down kernel
    float *y = nullptr;
};
size_t moe_few_act_ints(size_t m, size_t experts, size_t top);
int launch_moe_few(Ctx *ctx, const MoeFewCall &c, cudaStream_t st);

}  // namespace lbk
