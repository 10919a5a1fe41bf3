// Calls of the sequence mixers beside plain attention: latent attention (lbk_latent.cu) and linear recurrences
// (lbk_recur.cu). Rows are consecutive positions of one sequence (rows_of_seq >= 0, pos[0] the first one's position)
// or one new token of each sequence (rows_of_seq = -1, row t is sequence t at pos[t]), as in DenseEpi.
#pragma once

#include "lbk_dense.cuh"

namespace lbk {

// ---- rotation of neighbouring dimensions ------------------------------------------------------------
// Pair i is turned by position * freq[i]; cos and sin are multiplied by `factor`.
struct Rotation {
    const double *freq = nullptr;  // device, [dims / 2]
    int dims = 0;
    float factor = 1.0f;
};
// The frequencies base^(-2i/dims), on the host; with `yarn` the interpolation between a pair's own frequency and
// 1 / scale of it (ramp between the pairs that turn `fast` and `slow` times in `original` positions).
struct YarnScaling {
    bool on = false;
    double factor = 1.0, original = 1.0, fast = 1.0, slow = 1.0;
};
void rotation_frequencies(size_t dims, double base, const YarnScaling &yarn, double *freq, float *factor);

// ---- latent attention ---------------------------------------------------------------------------------
// A position caches one row of `pitch` values: the latent (kv_rank values, zeros up to kvp), then the rotated key part
// (rot_dim values, zeros up to rp).
struct LatentShape {
    size_t heads = 0, dim = 0, rot_dim = 0, vdim = 0, kv_rank = 0, q_rank = 0;
    size_t dp() const { return pad16(dim); }
    size_t rp() const { return pad16(rot_dim); }
    size_t kvp() const { return pad16(kv_rank); }
    size_t vp() const { return pad16(vdim); }
    size_t qp() const { return dp() + rp(); }                    // a query head as the projection leaves it
    size_t pitch() const { return dense_pitch(kvp() + rp()); }   // a cache row, and a query head against it
};
// z f32 [rows][ldz] = [query latent q_rank | latent kv_rank | key part rot_dim | gates]: the normed query latent to cq
// (compute type, pitch ldq); with `cache` also the normed latent and the rotated key part into the row's cache row.
struct LatentPrepCall {
    int compute = LBK_COMPUTE_BF16;
    LatentShape s;
    const float *z = nullptr;
    long ldz = 0;
    size_t rows = 0;
    int rows_of_seq = -1;
    const int *pos = nullptr;
    size_t cap = 0;
    const float *q_norm = nullptr, *kv_norm = nullptr;
    float eps = 0.0f;
    Rotation rot;
    void *cq = nullptr;
    long ldq = 0;
    void *cache = nullptr;  // [seq][cap][pitch]
};
int launch_latent_prep(Ctx *ctx, const LatentPrepCall &c, cudaStream_t st);

// Attention of `rows` queries over the cached latents. q [rows][heads][qp], not rotated yet (rotated in place by the
// expanding form). out [rows][heads * vdim], pitch ldo: softmax((q . k) * scale) v, times sigmoid(gate[t * ldg + h]).
//   absorbing form (any rows): W_uk^T q against the latents themselves, W_uv on the weighted latents
//   expanding form (prompt rows, bf16): keys and values of all `length` positions are written out per head first
struct LatentAttnCall {
    int compute = LBK_COMPUTE_BF16;
    LatentShape s;
    void *q = nullptr;
    size_t rows = 0;
    int rows_of_seq = -1;
    const int *pos = nullptr;
    size_t cap = 0;
    const void *cache = nullptr;
    DenseWeight uk, uv;             // [heads * dim][kv_rank], [heads * vdim][kv_rank]
    DenseWeight ukv;                // both, uk first (expanding form)
    float scale = 1.0f;
    Rotation rot;
    const float *gate = nullptr;
    long ldg = 0;
    void *ql = nullptr;             // absorbing form: [rows][heads][pitch] of the compute type, zeros past kvp + rot_dim
    float *scratch = nullptr;       // absorbing form: latent_scratch floats
    size_t splits = 0;              // slices of the keys that scratch was sized for
    size_t length = 0;              // expanding form: positions the sequence has after these rows
    void *ek = nullptr, *ev = nullptr;  // expanding form: [heads][ecap][dp], [heads][ecap][vp] bf16
    size_t ecap = 0;
    const int *zero = nullptr;      // a zero on the device
    void *out = nullptr;
    long ldo = 0;
};
size_t latent_splits(size_t cap);
size_t latent_scratch(const Ctx *ctx, size_t rows, const LatentShape &s, size_t splits);
bool latent_absorb_supported(const LatentShape &s);  // bf16; 32-bit has no such limit
bool latent_expand_supported(const LatentShape &s);
int launch_latent_absorbed(Ctx *ctx, const LatentAttnCall &c, cudaStream_t st);
int launch_latent_expanded(Ctx *ctx, const LatentAttnCall &c, cudaStream_t st);

// ---- linear recurrences -------------------------------------------------------------------------------
// A state S [vdim][dim] (f32) per head and sequence; a sequence at position 0 starts from zero.
//   plain:  S <- decay_h S + k v^T,                                     o = S^T q
//   delta:  S <- g S (per key channel); u = beta (v - S^T k); S <- S + k u^T;  o = S^T q
// x: rows of the compute type, pitch ldx, with q, k, v at the given columns (delta: before their short convolution).
struct RecurCall {
    int compute = LBK_COMPUTE_BF16;
    bool delta = false;
    size_t heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    const void *x = nullptr;
    long ldx = 0;
    int q_at = 0, k_at = 0, v_at = 0;
    size_t rows = 0;
    int rows_of_seq = -1;
    const int *pos = nullptr, *active = nullptr;  // active [seq]: 0: the sequence's state is left as it is (rows_of_seq = -1)
    size_t cap = 0;
    const float *decay = nullptr;        // plain: [heads]
    // delta
    int taps = 1;
    const float *conv = nullptr;         // [taps][channels], channels as in x from q_at on: q, k, v back to back
    void *ring = nullptr;                // [seq][taps][channels] of the compute type: the last inputs, by position modulo taps
    const float *a = nullptr;            // [rows][lda] f32, heads x dim: the projection inside softplus
    long lda = 0;
    const float *a_log = nullptr, *dt_bias = nullptr;  // [heads], [heads * dim]
    const float *b = nullptr;            // [rows][ldb]: logits of beta, one per head
    long ldb = 0;
    float *state = nullptr;              // [seq][heads][vdim][recur_pitch(dim)]
    float *records = nullptr;            // rows_of_seq >= 0: recur_record_floats
    size_t record_rows = 0;              // rows the records were sized for (more are done in several runs)
    float *o = nullptr;                  // [rows][heads * vdim]
    // delta, one token per sequence: instead of `a` the second halves of both low-rank projections (inputs at columns
    // a_at and g_at of x), and instead of o the gated norm per head (RMS over vdim, times norm_w, times sigmoid(gate))
    DenseWeight a2, g2;                  // [heads * dim][rank], [heads * vdim][rank]
    int a_at = 0, g_at = 0;
    const float *norm_w = nullptr;
    float eps = 0.0f;
    void *out = nullptr;                 // [rows][heads * vdim] of the compute type, pitch ldo
    long ldo = 0;
};
size_t recur_pitch(size_t dim);
size_t recur_record_floats(bool delta, size_t rows, size_t heads, size_t dim, size_t vdim);
constexpr size_t kRecurMaxDim = 256;
int launch_recurrence(Ctx *ctx, const RecurCall &c, cudaStream_t st);

// out[t][i] = o[t][i] / rms(its group) * w[i % group_w] * sigmoid(gate[t][i]); groups of `group` values. gate and out
// are rows of the compute type.
struct GatedNormCall {
    int compute = LBK_COMPUTE_BF16;
    const float *o = nullptr;
    size_t rows = 0, n = 0, group = 0;
    const float *w = nullptr;   // [group]
    const void *gate = nullptr;
    long ldg = 0;
    float eps = 0.0f;
    void *out = nullptr;
    long ldo = 0;
};
int launch_gated_norm(Ctx *ctx, const GatedNormCall &c, cudaStream_t st);

}  // namespace lbk
