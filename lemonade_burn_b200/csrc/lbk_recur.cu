// Linear recurrences: attention whose past is a matrix S [dim x vdim] per head instead of a list of keys.
//
//   plain   S <- decay S + k v^T;  o = S^T q                     (decay: a constant of the head)
//   delta   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q      (g: per token, head and key channel)
//
// The state and everything that enters it are f32 on the FMA pipes; nothing of a recurrence is rounded to 16 bits. Prompt
// rows are taken eight at a time. With S the state in front of eight tokens, G_i the product of their decays up to and
// including token i, and "after j" the product of those behind token j:
//
//   a_i = S^T (k_i G_i)      b_i = S^T (q_i G_i)
//   u_i = beta_i (v_i - a_i - sum_{j<i} c_ij u_j)       c_ij = k_i . (k_j x decays j+1 .. i)       (plain: u_i = v_i)
//   o_i = b_i + sum_{j<=i} p_ij u_j                     p_ij = q_i . (k_j x decays j+1 .. i)
//   S  <- G_7 S + sum_j (k_j x decays after j) u_j^T
//
// which is the recurrence itself, reordered: one multiplication of the state by decays instead of eight and products of
// at most eight decays (never a quotient, so strong decays underflow to zero as they should). The equations for u are a
// triangular system of the eight tokens; its inverse T (u = T (v - a)) is worked out ahead. Kernels:
//
//   recur_prep_kernel   one block per (eight tokens, head): q, k, v as they are or, for delta, short convolution + silu, unit
//                       vectors, decays and step sizes; writes one record per (eight tokens, head) with the vectors
//                       and numbers above. Every token block is independent of every other.
//   recur_walk_kernel   one block per (head, slice of value columns) walks the records in order. A warp holds four columns
//                       of S in registers, dim / 32 values of each a lane (packed pairs for the two-wide FMA), so a vector
//                       read from shared memory serves four columns. The dots over the 32 lanes meet by transposing
//                       shuffles: lane l ends up with those of column l / 8 and token l % 8. Every lane keeps its
//                       partial dots in an order of its own, slot s holding dot s XOR l, so that each step of the
//                       transposition adds a received value to a register without choosing. A producer lane brings the
//                       records into a ring of shared memory with bulk copies.
//   recur_step_kernel   decode: one block per (head, sequence) does all of a token: convolution, both low-rank second
//                       halves, unit vectors, decays, the state (on its way from memory meanwhile), the read-out and, per
//                       head, its gated norm.
//   gated_norm_kernel   the read-out divided by its root mean square per group, times a weight and sigmoid(gate).
//
// A sequence at position 0 starts from a zero state whatever the buffer holds, so a slot that is used again needs no
// clearing. Convolution inputs that later tokens need stay in a ring by position, one place more than are read; the walk
// stores them (after every prep block of the pass has read the old ones).
#include "lbk_dense_dev.cuh"
#include "lbk_mixers.cuh"
#include "lbk_ptx.cuh"

namespace lbk {

namespace {

constexpr int kTok = 8;             // tokens per record
constexpr int kPrepThreads = 128;
constexpr int kScal = 2 * kTok * kTok;  // numbers of a record: T, then p, eight by eight
constexpr int kMaxWarps = 8;        // warps that hold columns, four columns each
constexpr int kMaxStages = 12;
constexpr uint32_t kWaitLimit = 1u << 22;

struct RecurParams {
    const void *x;
    long ldx;
    int q_at, k_at, v_at, heads, kv_heads, dim, vdim, dp, vp;
    int n, rows_of_seq, row0, blocks, cap, taps, last, total;
    const int *pos, *active;
    const float *decay;
    const float *conv;              // [taps][channels]
    void *ring;
    int channels;
    const float *a;
    long lda;
    const float *a_log, *dt_bias, *b;
    long ldb;
    float *state, *records;
    int rec;                        // floats of a record
    float *o;
    int stages, warps;
    int *err_word;
    // recur_step_kernel
    const uint16_t *a2, *g2;
    int a2_pitch, g2_pitch, a_at, g_at, a_rank, g_rank;
    const float *norm_w;
    float eps;
    void *out;
    long ldo;
};

__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }
template <typename T>
__device__ __forceinline__ float act(float z) { return dense::silu<sizeof(T) == 4>(z); }
__device__ __forceinline__ float decay_of(float rate, float z) { return expf(-rate * softplus(z)); }

// Sums of N (a power of two, at most 32) values over a warp: lane l gets the total of value l % N.
template <int N>
__device__ __forceinline__ float warp_sums(float (&v)[N], int lane) {
#pragma unroll
    for (int w = N / 2; w >= 1; w >>= 1) {
        const bool up = (lane & w) != 0;
#pragma unroll
        for (int i = 0; i < w; ++i) v[i] = (up ? v[i + w] : v[i]) + __shfl_xor_sync(0xffffffffu, up ? v[i] : v[i + w], w);
    }
    float t = v[0];
#pragma unroll
    for (int w = N; w < 32; w <<= 1) t += __shfl_xor_sync(0xffffffffu, t, w);
    return t;
}

// The eight tokens' values of one channel (`col`: row 0 of the pass; `cc`: the channel of the convolution): as they are, or
// convolved over `taps` inputs. Rows in front of the pass come from the ring, positions in front of 0 are zeros.
template <typename T, bool DELTA>
__device__ __forceinline__ void channel_values(const RecurParams &p, const T *col, int cc, int row0, int cnt, int pos0, int taps, float (&y)[kTok]) {
    const T *at = col + static_cast<size_t>(row0) * p.ldx;
    if (!DELTA) {
#pragma unroll
        for (int i = 0; i < kTok; ++i) y[i] = i < cnt ? dense::get(at + i * p.ldx) : 0.0f;
        return;
    }
    const int back = taps - 1;
    const float *c = p.conv + cc;
    auto convolve = [&](auto input) {
        float w[kTok];
#pragma unroll
        for (int i = 0; i < kTok; ++i) {
            w[i] = input(i - back);
            y[i] = w[i] * c[0];
        }
#pragma unroll
        for (int j = 1; j < taps; ++j) {
#pragma unroll
            for (int i = 0; i + 1 < kTok; ++i) w[i] = w[i + 1];
            w[kTok - 1] = input(kTok - 1 - back + j);
            const float cj = c[static_cast<size_t>(j) * p.channels];
#pragma unroll
            for (int i = 0; i < kTok; ++i) y[i] = fmaf(w[i], cj, y[i]);
        }
    };
    if (row0 >= back && cnt == kTok) {  // every input is a row of this pass
        const T *first = at - static_cast<long>(back) * p.ldx;
        convolve([&](int r) { return dense::get(first + (r + back) * p.ldx); });
    } else {
        convolve([&](int r) -> float {  // row row0 + r
            if (r >= cnt) return 0.0f;
            if (row0 + r >= 0) return dense::get(at + r * p.ldx);
            const int ps = pos0 + row0 + r;
            return ps >= 0 ? dense::get(static_cast<const T *>(p.ring) + (static_cast<size_t>(p.rows_of_seq) * taps + ps % taps) * p.channels + cc) : 0.0f;
        });
    }
#pragma unroll
    for (int i = 0; i < kTok; ++i) y[i] = i < cnt ? act<T>(y[i]) : 0.0f;
}

// NB: dimensions a thread takes (dp / 128, at least 1); TAPS: 0 for any number
template <typename T, bool DELTA, int NB, int TAPS>
__global__ void __launch_bounds__(kPrepThreads) recur_prep_kernel(const RecurParams p) {
    ptx::pdl_trigger();
    ptx::pdl_wait();
    __shared__ float s_red[4][64];
    __shared__ float s_c[kTok][kTok];
    const int h = blockIdx.x, blk = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int row0 = p.row0 + blk * kTok;                  // row of token 0 of this record
    const int cnt = min(kTok, p.row0 + p.n - row0), taps = TAPS ? TAPS : p.taps;
    const int pos0 = p.pos[0];                             // position of row 0 of the pass
    if (pos0 < 0 || pos0 + p.total > p.cap) {
        if (tid == 0) atomicExch(p.err_word, 7);
        return;
    }
    const T *x = static_cast<const T *>(p.x);
    float *rec = p.records + static_cast<size_t>(h * p.blocks + blk) * p.rec;
    const int kvh = h / (p.heads / p.kv_heads);
    auto values = [&](int at, int ch, float (&y)[kTok]) { channel_values<T, DELTA>(p, x + at + ch, at - p.q_at + ch, row0, cnt, pos0, taps, y); };
    float *rk = rec, *rq = rec + (DELTA ? kTok : 0) * p.dp, *rh = rq + kTok * p.dp, *rg = rh + kTok * p.dp, *rs = rg + p.dp, *rv = rs + kScal;
    float q[NB][kTok], k[NB][kTok], g[NB][kTok];
#pragma unroll
    for (int b = 0; b < NB; ++b) {
        const int d = tid + b * kPrepThreads;
#pragma unroll
        for (int i = 0; i < kTok; ++i) q[b][i] = k[b][i] = 0.0f, g[b][i] = 1.0f;
        if (d < p.dim) {
            if (DELTA) {
                const float *a = p.a + static_cast<size_t>(row0) * p.lda + h * p.dim + d;
#pragma unroll
                for (int i = 0; i < kTok; ++i) g[b][i] = i < cnt ? a[i * p.lda] : 0.0f;
            }
            values(p.q_at, kvh * p.dim + d, q[b]);
            values(p.k_at, kvh * p.dim + d, k[b]);
        }
    }
    for (int c = tid; c < p.vp; c += kPrepThreads) {
        float v[kTok];
#pragma unroll
        for (int i = 0; i < kTok; ++i) v[i] = 0.0f;
        if (c < p.vdim) values(p.v_at, h * p.vdim + c, v);
#pragma unroll
        for (int i = 0; i < kTok; ++i) rv[i * p.vp + c] = v[i];
    }
    if (DELTA) {
        float ss[2 * kTok];
#pragma unroll
        for (int i = 0; i < 2 * kTok; ++i) ss[i] = 0.0f;
#pragma unroll
        for (int b = 0; b < NB; ++b)
#pragma unroll
            for (int i = 0; i < kTok; ++i) {
                ss[i] = fmaf(q[b][i], q[b][i], ss[i]);
                ss[kTok + i] = fmaf(k[b][i], k[b][i], ss[kTok + i]);
            }
        const float t = warp_sums(ss, lane);
        if (lane < 2 * kTok) s_red[warp][lane] = t;
        const float rate = expf(p.a_log[h]);
#pragma unroll
        for (int b = 0; b < NB; ++b) {
            const int d = tid + b * kPrepThreads;
            const float bias = d < p.dim ? p.dt_bias[h * p.dim + d] : 0.0f;
#pragma unroll
            for (int i = 0; i < kTok; ++i) g[b][i] = d < p.dim && i < cnt ? decay_of(rate, g[b][i] + bias) : 1.0f;
        }
        __syncthreads();
        if (tid < 2 * kTok) {                              // the factors that make unit vectors
            const float sum = (s_red[0][tid] + s_red[1][tid]) + (s_red[2][tid] + s_red[3][tid]);
            s_c[0][tid] = (tid < kTok ? 1.0f / sqrtf(static_cast<float>(p.dim)) : 1.0f) / sqrtf(sum + 1e-6f);
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < kTok; ++i) {
            const float fq = s_c[0][i], fk = s_c[1][i];
#pragma unroll
            for (int b = 0; b < NB; ++b) {
                q[b][i] *= fq;
                k[b][i] *= fk;
            }
        }
        __syncthreads();
    } else {
        const float decay = p.decay[h];
#pragma unroll
        for (int b = 0; b < NB; ++b)
#pragma unroll
            for (int i = 0; i < kTok; ++i) g[b][i] = i < cnt ? decay : 1.0f;
    }
    // the record
#pragma unroll
    for (int b = 0; b < NB; ++b) {
        const int d = tid + b * kPrepThreads;
        if (d < p.dp) {
            float after = 1.0f, upto = 1.0f;
#pragma unroll
            for (int i = 0; i < kTok; ++i) {
                upto *= g[b][i];
                if (DELTA) rk[i * p.dp + d] = k[b][i] * upto;
                rq[i * p.dp + d] = q[b][i] * upto;
            }
            rg[d] = upto;
#pragma unroll
            for (int j = kTok - 1; j >= 0; --j) {
                rh[j * p.dp + d] = k[b][j] * after;
                after *= g[b][j];
            }
        }
    }
    // dots of pairs (i, j): 32 at a time; j <= i with q_i first (36), then j < i with k_i (28)
#pragma unroll
    for (int part = 0; part < 2; ++part) {
        float dots[32];
#pragma unroll
        for (int e = 0; e < 32; ++e) dots[e] = 0.0f;
#pragma unroll
        for (int b = 0; b < NB; ++b) {
#pragma unroll
            for (int i = 0; i < kTok; ++i) {
                float f = 1.0f;
#pragma unroll
                for (int j = i; j >= 0; --j) {
                    const int ep = i * (i + 1) / 2 + j, ec = 36 + i * (i - 1) / 2 + j;
                    if (ep >= part * 32 && ep < part * 32 + 32) dots[ep & 31] = fmaf(q[b][i] * f, k[b][j], dots[ep & 31]);
                    if (DELTA && j < i && ec >= part * 32 && ec < part * 32 + 32) dots[ec & 31] = fmaf(k[b][i] * f, k[b][j], dots[ec & 31]);
                    f *= g[b][j];
                }
            }
        }
        const float t = warp_sums(dots, lane);
        s_red[warp][part * 32 + lane] = t;
    }
    __syncthreads();
    if (tid < kTok * kTok) {
        const int i = tid >> 3, j = tid & 7;
        auto sum = [&](int e) { return (s_red[0][e] + s_red[1][e]) + (s_red[2][e] + s_red[3][e]); };
        rs[kTok * kTok + tid] = j <= i ? sum(i * (i + 1) / 2 + j) : 0.0f;
        s_c[i][j] = DELTA && j < i ? sum(36 + i * (i - 1) / 2 + j) : 0.0f;
        if (!DELTA) rs[tid] = i == j ? 1.0f : 0.0f;
    }
    if (DELTA) {
        __syncthreads();
        if (tid < kTok) {                                  // column `tid` of T: forward substitution
            float t[kTok];
#pragma unroll
            for (int i = 0; i < kTok; ++i) {
                const float beta = i < cnt ? dense::sigmoid(p.b[static_cast<size_t>(row0 + i) * p.ldb + h]) : 0.0f;
                float v = i == tid ? 1.0f : 0.0f;
#pragma unroll
                for (int j = 0; j < i; ++j) v = fmaf(-s_c[i][j], t[j], v);
                t[i] = beta * v;
                rs[i * kTok + tid] = t[i];
            }
        }
    }
}

// ---- the walk ---------------------------------------------------------------------------------------
using u64 = unsigned long long;
__device__ __forceinline__ u64 fma2(u64 a, u64 b, u64 c) {
    u64 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ u64 mul2(u64 a, u64 b) {
    u64 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ u64 pack2(float x, float y) {
    u64 d;
    asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(x), "f"(y));
    return d;
}
__device__ __forceinline__ float sum2(u64 a) {
    float x, y;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(a));
    return x + y;
}
__device__ __forceinline__ void bulk_load(uint32_t dst, const void *src, uint32_t bytes, uint32_t bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst), "l"(src), "r"(bytes), "r"(bar) : "memory");
}
// A lane's share of a vector of 64 P values: pairs at 2 lane (P = 1), quadruples at 4 lane + 128 j else.
template <int P>
__device__ __forceinline__ void share(const float *v, int lane, u64 (&r)[P]) {
    if (P == 1) {
        r[0] = *reinterpret_cast<const u64 *>(v + 2 * lane);
    } else {
#pragma unroll
        for (int j = 0; j < P / 2; ++j) {
            const ulonglong2 t = *reinterpret_cast<const ulonglong2 *>(v + 128 * j + 4 * lane);
            r[2 * j] = t.x;
            r[2 * j + 1] = t.y;
        }
    }
}
template <int P>
__device__ __forceinline__ void unshare(float *v, int lane, const u64 (&r)[P]) {
    if (P == 1) {
        *reinterpret_cast<u64 *>(v + 2 * lane) = r[0];
    } else {
#pragma unroll
        for (int j = 0; j < P / 2; ++j) *reinterpret_cast<ulonglong2 *>(v + 128 * j + 4 * lane) = make_ulonglong2(r[2 * j], r[2 * j + 1]);
    }
}
template <int P>
__device__ __forceinline__ float dot(const u64 (&a)[P], const u64 (&b)[P]) {
    u64 t = mul2(a[0], b[0]);
#pragma unroll
    for (int i = 1; i < P; ++i) t = fma2(a[i], b[i], t);
    return sum2(t);
}

// P: packed pairs of a column per lane (dp = 64 P). Slot s of a lane holds column s XOR (lane / 8) of the warp's four.
template <typename T, bool DELTA, int P>
__global__ void __launch_bounds__((kMaxWarps + 1) * 32) recur_walk_kernel(const RecurParams p) {
    extern __shared__ __align__(16) uint8_t rc_smem[];
    __shared__ __align__(8) uint64_t s_bar[2 * kMaxStages];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int h = blockIdx.y, slice = blockIdx.x, seq = p.rows_of_seq;
    const uint32_t bar0 = ptx::smem_u32(s_bar), ring0 = ptx::smem_u32(rc_smem);
    const uint32_t bytes = static_cast<uint32_t>(p.rec) * 4;
    if (tid == 0) {
        for (int s = 0; s < p.stages; ++s) {
            ptx::mbar_init(bar0 + s * 8, 1);
            ptx::mbar_init(bar0 + (kMaxStages + s) * 8, p.warps);
        }
        ptx::fence_barrier_init();
    }
    __syncthreads();
    ptx::pdl_trigger();
    ptx::pdl_wait();
    const int pos_first = p.pos[0];
    const bool fits = pos_first >= 0 && pos_first + p.total <= p.cap;   // the prep kernel has flagged it
    const int blocks = fits ? p.blocks : 0;
    if (warp == p.warps) {
        if (lane == 0) {
            const float *rec = p.records + static_cast<size_t>(h * p.blocks) * p.rec;
            for (int b = 0; b < blocks; ++b) {
                const int s = b % p.stages, round = b / p.stages;
                if (round > 0 && !ptx::mbar_wait(bar0 + (kMaxStages + s) * 8, (round - 1) & 1, kWaitLimit)) {
                    atomicExch(p.err_word, 5);
                    break;
                }
                ptx::mbar_arrive_expect_tx(bar0 + s * 8, bytes);
                bulk_load(ring0 + s * bytes, rec + static_cast<size_t>(b) * p.rec, bytes, bar0 + s * 8);
            }
        }
    } else {
        const int cg = lane >> 3, col0 = (slice * p.warps + warp) * 4, col = col0 + cg, tk = lane & 7;  // the lane's own column and token
        float *st = p.state + static_cast<size_t>(seq * p.heads + h) * p.vdim * p.dp;
        u64 S[4][P];
#pragma unroll
        for (int s = 0; s < 4; ++s) {
#pragma unroll
            for (int j = 0; j < P; ++j) S[s][j] = 0;
            if (pos_first + p.row0 > 0 && col0 + (s ^ cg) < p.vdim) share<P>(st + static_cast<size_t>(col0 + (s ^ cg)) * p.dp, lane, S[s]);
        }
        bool ok = true;
        int s = 0, phase = 0;
        for (int b = 0; b < blocks; ++b) {
            if (!__all_sync(0xffffffffu, ptx::mbar_wait(bar0 + s * 8, phase, kWaitLimit))) {
                ok = false;
                break;
            }
            const float *rec = reinterpret_cast<const float *>(rc_smem + static_cast<size_t>(s) * bytes);
            const float *rk = rec, *rq = rec + (DELTA ? kTok : 0) * 64 * P, *rh = rq + kTok * 64 * P, *rg = rh + kTok * 64 * P, *rs = rg + 64 * P, *rv = rs + kScal;
            // dots of eight tokens' vectors with the four columns; the lane's own token and column
            auto dots = [&](const float *rows) -> float {
                float r[kTok];
#pragma unroll
                for (int e = 0; e < kTok; ++e) {
                    u64 w[P];
                    share<P>(rows + (e ^ tk) * 64 * P, lane, w);
                    float v0 = dot<P>(w, S[0]), v1 = dot<P>(w, S[1]);
                    const float v2 = dot<P>(w, S[2]), v3 = dot<P>(w, S[3]);
                    v0 += __shfl_xor_sync(0xffffffffu, v2, 16);
                    v1 += __shfl_xor_sync(0xffffffffu, v3, 16);
                    r[e] = v0 + __shfl_xor_sync(0xffffffffu, v1, 8);
                }
#pragma unroll
                for (int w = kTok / 2; w >= 1; w >>= 1)
#pragma unroll
                    for (int e = 0; e < w; ++e) r[e] += __shfl_xor_sync(0xffffffffu, r[e + w], w);
                return r[0];
            };
            auto times = [&](const float *row, const float (&v)[kTok]) -> float {  // eight numbers of shared memory . v
                const float4 a = *reinterpret_cast<const float4 *>(row), c = *reinterpret_cast<const float4 *>(row + 4);
                return fmaf(a.x, v[0], fmaf(a.y, v[1], fmaf(a.z, v[2], a.w * v[3]))) + fmaf(c.x, v[4], fmaf(c.y, v[5], fmaf(c.z, v[6], c.w * v[7])));
            };
            float mine = rv[tk * p.vp + min(col, p.vdim - 1)], u[kTok];
            float read = 0.0f;
            if (DELTA) {
                mine -= dots(rk);
                read = dots(rq);
                float t[kTok];
#pragma unroll
                for (int j = 0; j < kTok; ++j) t[j] = __shfl_sync(0xffffffffu, mine, (lane & 24) | j);
                mine = times(rs + kTok * tk, t);
            } else {
                read = dots(rq);
            }
#pragma unroll
            for (int j = 0; j < kTok; ++j) u[j] = __shfl_sync(0xffffffffu, mine, (lane & 24) | j);
            if (b * kTok + tk < p.n && col < p.vdim)
                p.o[(static_cast<size_t>(p.row0 + b * kTok + tk) * p.heads + h) * p.vdim + col] = read + times(rs + kTok * kTok + kTok * tk, u);
            u64 g[P];
            share<P>(rg, lane, g);
#pragma unroll
            for (int c = 0; c < 4; ++c)
#pragma unroll
                for (int j = 0; j < P; ++j) S[c][j] = mul2(g[j], S[c][j]);
#pragma unroll
            for (int i = 0; i < kTok; ++i) {
                u64 w[P];
                share<P>(rh + i * 64 * P, lane, w);
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    const float uc = c ? __shfl_xor_sync(0xffffffffu, u[i], 8 * c) : u[i];
                    const u64 uu = pack2(uc, uc);
#pragma unroll
                    for (int j = 0; j < P; ++j) S[c][j] = fma2(w[j], uu, S[c][j]);
                }
            }
            __syncwarp();
            if (lane == 0) ptx::mbar_arrive(bar0 + (kMaxStages + s) * 8);
            if (++s == p.stages) {
                s = 0;
                phase ^= 1;
            }
        }
        if (!ok && lane == 0) atomicExch(p.err_word, 5);
        if (ok && fits) {
#pragma unroll
            for (int c = 0; c < 4; ++c)
                if (col0 + (c ^ cg) < p.vdim) unshare<P>(st + static_cast<size_t>(col0 + (c ^ cg)) * p.dp, lane, S[c]);
            if (DELTA && slice == 0 && p.last && p.taps > 1) {
                // the inputs later tokens will convolve with: the last taps - 1 of this pass, this head's channels
                const T *x = static_cast<const T *>(p.x);
                const int group = p.heads / p.kv_heads, qk = h % group == 0 ? 2 * p.dim : 0, all = qk + p.vdim;
                const int rows = min(p.taps - 1, p.total);
                for (int e = tid; e < rows * all; e += p.warps * 32) {
                    const int r = e / all, c = e - r * all;
                    const int at = c < qk ? (c < p.dim ? p.q_at : p.k_at - p.dim) + (h / group) * p.dim + c : p.v_at + h * p.vdim + c - qk;
                    const int row = p.total - rows + r;
                    static_cast<T *>(p.ring)[(static_cast<size_t>(seq) * p.taps + (pos_first + row) % p.taps) * p.channels + at - p.q_at] = x[static_cast<size_t>(row) * p.ldx + at];
                }
            }
        }
    }
}

// ---- one token --------------------------------------------------------------------------------------------
constexpr int kStepWarps = 16, kStepThreads = kStepWarps * 32;

// `rows` rows of W (bf16, [rows][pitch]) times the vector x (rank values, any alignment): four threads a row, the result of
// row r to out(r, value) in its first thread.
template <typename T, typename F>
__device__ __forceinline__ void low_rank(const uint16_t *w, int pitch, int rank, const T *x, int rows, float *s_x, F &&out) {
    const int tid = threadIdx.x;
    __syncthreads();
    for (int i = tid; i < pitch; i += kStepThreads) s_x[i] = i < rank ? dense::get(x + i) : 0.0f;
    __syncthreads();
    for (int r0 = 0; r0 < rows; r0 += kStepThreads / 4) {
        const int r = r0 + (tid >> 2), part = tid & 3;
        float acc = 0.0f;
        if (r < rows)
            for (int c = part * 8; c < pitch; c += 32) {
                const uint4 v = *reinterpret_cast<const uint4 *>(w + static_cast<size_t>(r) * pitch + c);
                const uint32_t wv[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    acc = fmaf(__uint_as_float(wv[e] << 16), s_x[c + 2 * e], acc);
                    acc = fmaf(__uint_as_float(wv[e] & 0xffff0000u), s_x[c + 2 * e + 1], acc);
                }
            }
        acc += __shfl_xor_sync(0xffffffffu, acc, 1);
        acc += __shfl_xor_sync(0xffffffffu, acc, 2);
        if (r < rows && part == 0) out(r, acc);
    }
}

// A warp takes eight columns of S at a time. Slot s of a lane holds column s XOR (lane / 4) of the eight.
template <typename T, bool DELTA, int P>
__global__ void __launch_bounds__(kStepThreads, 1) recur_step_kernel(const RecurParams p) {
    extern __shared__ __align__(16) float rs_smem[];
    __shared__ float s_red[32], s_sum[4];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.x, seq = blockIdx.y;
    float *s_k = rs_smem, *s_q = s_k + 64 * P, *s_kg = s_q + 64 * P, *s_qg = s_kg + 64 * P, *s_g = s_qg + 64 * P, *s_v = s_g + 64 * P;
    float *s_o = s_v + p.vp, *s_gate = s_o + p.vp, *s_x = s_gate + p.vp;
    ptx::pdl_trigger();
    ptx::pdl_wait();
    const int pos = p.pos[seq];
    if (pos < 0 || pos >= p.cap) {
        if (tid == 0) atomicExch(p.err_word, 7);
        return;
    }
    const bool keep = !p.active || p.active[seq] != 0;
    float *st = p.state + static_cast<size_t>(seq * p.heads + h) * p.vdim * p.dp;
    const int cg = lane >> 2;
    u64 S[8][P];
    auto load = [&](int col0) {
#pragma unroll
        for (int s = 0; s < 8; ++s) {
#pragma unroll
            for (int j = 0; j < P; ++j) S[s][j] = 0;
            if (pos > 0 && col0 + (s ^ cg) < p.vdim) share<P>(st + static_cast<size_t>(col0 + (s ^ cg)) * p.dp, lane, S[s]);
        }
    };
    load(warp * 8);  // on its way while the token's vectors are worked out
    const T *x = static_cast<const T *>(p.x) + static_cast<size_t>(seq) * p.ldx;
    const int group = p.heads / p.kv_heads, kvh = h / group;
    for (int e = tid; e < 128 * P + p.vp; e += kStepThreads) {
        const int which = e < 64 * P ? 0 : e < 128 * P ? 1 : 2, d = which == 0 ? e : which == 1 ? e - 64 * P : e - 128 * P;
        float v = 0.0f;
        if (d < (which < 2 ? p.dim : p.vdim)) {
            const int at = (which == 0 ? p.q_at + kvh * p.dim : which == 1 ? p.k_at + kvh * p.dim : p.v_at + h * p.vdim) + d;
            v = dense::get(x + at);
            if (DELTA) {
                const int cc = at - p.q_at;
                T *ring = static_cast<T *>(p.ring) + static_cast<size_t>(seq) * p.taps * p.channels + cc;
                float y = v * p.conv[static_cast<size_t>(p.taps - 1) * p.channels + cc];
                for (int back = 1; back < p.taps; ++back)
                    if (pos - back >= 0)
                        y = fmaf(dense::get(ring + static_cast<size_t>((pos - back) % p.taps) * p.channels), p.conv[static_cast<size_t>(p.taps - 1 - back) * p.channels + cc], y);
                // the place of this token is not one that is read now; q and k belong to the first head of their group
                if (keep && (which == 2 || h % group == 0)) ring[static_cast<size_t>(pos % p.taps) * p.channels] = x[at];
                v = act<T>(y);
            }
        }
        (which == 0 ? s_q : which == 1 ? s_k : s_v)[d] = v;
    }
    if (DELTA) {
        const float rate = expf(p.a_log[h]);
        auto decay = [&](int d, float z) { s_g[d] = decay_of(rate, z + p.dt_bias[h * p.dim + d]); };
        if (p.a2) {
            low_rank(p.a2 + static_cast<size_t>(h) * p.dim * p.a2_pitch, p.a2_pitch, p.a_rank, x + p.a_at, p.dim, s_x, decay);
            low_rank(p.g2 + static_cast<size_t>(h) * p.vdim * p.g2_pitch, p.g2_pitch, p.g_rank, x + p.g_at, p.vdim, s_x, [&](int d, float z) { s_gate[d] = dense::sigmoid(z); });
        } else {
            for (int d = tid; d < p.dim; d += kStepThreads) decay(d, p.a[static_cast<size_t>(seq) * p.lda + h * p.dim + d]);
        }
        for (int d = p.dim + tid; d < 64 * P; d += kStepThreads) s_g[d] = 1.0f;
    } else {
        for (int d = tid; d < 64 * P; d += kStepThreads) s_g[d] = p.decay[h];
    }
    __syncthreads();
    if (warp < 3) {  // |q|^2, |k|^2, q . k
        const float *l = warp == 1 ? s_k : s_q, *r = warp == 0 ? s_q : s_k;
        float t = 0.0f;
        for (int d = lane; d < 64 * P; d += 32) t = fmaf(l[d], r[d], t);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) t += __shfl_xor_sync(0xffffffffu, t, o);
        if (lane == 0) s_sum[warp] = t;
    }
    __syncthreads();
    const float fq = DELTA ? 1.0f / sqrtf(static_cast<float>(p.dim)) / sqrtf(s_sum[0] + 1e-6f) : 1.0f, fk = DELTA ? 1.0f / sqrtf(s_sum[1] + 1e-6f) : 1.0f;
    const float qk = s_sum[2] * fq * fk, beta = DELTA ? dense::sigmoid(p.b[static_cast<size_t>(seq) * p.ldb + h]) : 1.0f;
    for (int d = tid; d < 64 * P; d += kStepThreads) {
        const float k = s_k[d] * fk, g = s_g[d];
        s_k[d] = k;
        s_kg[d] = k * g;
        s_qg[d] = s_q[d] * fq * g;
    }
    __syncthreads();
    u64 w[P], wg[P], g[P], kk[P];
    const int up = lane >> 1 & 1;
    share<P>(up ? s_qg : s_kg, lane, w);   // slot 0 of the lane's two dots
    share<P>(up ? s_kg : s_qg, lane, wg);
    share<P>(s_g, lane, g);
    share<P>(s_k, lane, kk);
    for (int col0 = warp * 8; col0 < p.vdim; col0 += kStepWarps * 8) {
        if (col0 != warp * 8) load(col0);
        float r[8];
        if (DELTA) {
#pragma unroll
            for (int s = 0; s < 8; ++s) {
                r[s] = dot<P>(w, S[s]);
                r[s] += __shfl_xor_sync(0xffffffffu, dot<P>(wg, S[s]), 2);
            }
        } else {
#pragma unroll
            for (int s = 0; s < 8; ++s) r[s] = dot<P>(up ? w : wg, S[s]);
        }
#pragma unroll
        for (int c = 4; c >= 1; c >>= 1)
#pragma unroll
            for (int s = 0; s < c; ++s) r[s] += __shfl_xor_sync(0xffffffffu, r[s + c], 4 * c);
        float t = r[0] + __shfl_xor_sync(0xffffffffu, r[0], 1), u, b;
        const int col = col0 + cg;
        const float v = s_v[min(col, p.vdim - 1)];
        if (DELTA) {
            const float other = __shfl_xor_sync(0xffffffffu, t, 2);
            u = beta * (v - (up ? other : t));
            b = up ? t : other;
        } else {
            b = t + __shfl_xor_sync(0xffffffffu, t, 2);
            u = v;
        }
        if ((lane & 3) == 0 && col < p.vdim) s_o[col] = fmaf(qk, u, b);
        if (keep) {
#pragma unroll
            for (int s = 0; s < 8; ++s) {
                const float us = s ? __shfl_xor_sync(0xffffffffu, u, 4 * s) : u;
                const u64 uu = pack2(us, us);
#pragma unroll
                for (int j = 0; j < P; ++j) S[s][j] = fma2(kk[j], uu, mul2(g[j], S[s][j]));
                if (col0 + (s ^ cg) < p.vdim) unshare<P>(st + static_cast<size_t>(col0 + (s ^ cg)) * p.dp, lane, S[s]);
            }
        }
    }
    __syncthreads();
    if (DELTA && p.out) {
        float ss = 0.0f;
        for (int c = tid; c < p.vdim; c += kStepThreads) ss = fmaf(s_o[c], s_o[c], ss);
        const float r = 1.0f / sqrtf(dense::block_sum<kStepThreads>(ss, s_red) / static_cast<float>(p.vdim) + p.eps);
        T *out = static_cast<T *>(p.out) + static_cast<size_t>(seq) * p.ldo + static_cast<size_t>(h) * p.vdim;
        for (int c = tid; c < p.vdim; c += kStepThreads) dense::put(out + c, s_o[c] * r * p.norm_w[c] * s_gate[c]);
    } else {
        for (int c = tid; c < p.vdim; c += kStepThreads) p.o[(static_cast<size_t>(seq) * p.heads + h) * p.vdim + c] = s_o[c];
    }
}

// ---- gated norm -----------------------------------------------------------------------------------------
struct GatedParams {
    const float *o, *w;
    const void *gate;
    void *out;
    long ldg, ldo;
    int n, group;
    float eps;
};
// a warp per group of up to 32 * 32 values
template <typename T>
__global__ void __launch_bounds__(256) gated_norm_warp_kernel(const GatedParams p) {
    ptx::pdl_trigger();
    ptx::pdl_wait();
    const int lane = threadIdx.x & 31, g = blockIdx.x * 8 + (threadIdx.x >> 5);
    const size_t row = blockIdx.y;
    if (g * p.group >= p.n) return;
    const float *o = p.o + row * p.n + static_cast<size_t>(g) * p.group;
    float ss = 0.0f;
    for (int i = lane; i < p.group; i += 32) ss = fmaf(o[i], o[i], ss);
#pragma unroll
    for (int s = 16; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
    const float r = 1.0f / sqrtf(ss / static_cast<float>(p.group) + p.eps);
    const T *gate = static_cast<const T *>(p.gate) + row * p.ldg + static_cast<size_t>(g) * p.group;
    T *out = static_cast<T *>(p.out) + row * p.ldo + static_cast<size_t>(g) * p.group;
    for (int i = lane; i < p.group; i += 32) dense::put(out + i, o[i] * r * p.w[i] * dense::sigmoid(dense::get(gate + i)));
}
// a block per group
template <typename T>
__global__ void __launch_bounds__(512) gated_norm_block_kernel(const GatedParams p) {
    ptx::pdl_trigger();
    ptx::pdl_wait();
    __shared__ float s_red[32];
    const size_t row = blockIdx.y, g0 = static_cast<size_t>(blockIdx.x) * p.group;
    const float *o = p.o + row * p.n + g0;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < p.group; i += 512) ss = fmaf(o[i], o[i], ss);
    const float r = 1.0f / sqrtf(dense::block_sum<512>(ss, s_red) / static_cast<float>(p.group) + p.eps);
    const T *gate = static_cast<const T *>(p.gate) + row * p.ldg + g0;
    T *out = static_cast<T *>(p.out) + row * p.ldo + g0;
    for (int i = threadIdx.x; i < p.group; i += 512) dense::put(out + i, o[i] * r * p.w[i] * dense::sigmoid(dense::get(gate + i)));
}

__device__ __forceinline__ float4 get4(const float *p) { return *reinterpret_cast<const float4 *>(p); }
__device__ __forceinline__ float4 get4(const uint16_t *p) {
    const uint2 b = *reinterpret_cast<const uint2 *>(p);
    return make_float4(__uint_as_float(b.x << 16), __uint_as_float(b.x & 0xffff0000u), __uint_as_float(b.y << 16), __uint_as_float(b.y & 0xffff0000u));
}
__device__ __forceinline__ float gate_of(const float *, float z) { return dense::sigmoid(z); }
__device__ __forceinline__ float gate_of(const uint16_t *, float z) { return __fdividef(1.0f, 1.0f + __expf(-z)); }
// The same with four neighbouring values a thread, held in registers between the sum and the product: a block (LANES = 256)
// or a warp (32, eight groups a block) per group of up to 4 LANES NV values.
template <typename T, int LANES, int NV>
__global__ void __launch_bounds__(256) gated_norm_vec_kernel(const GatedParams p) {
    ptx::pdl_trigger();
    ptx::pdl_wait();
    __shared__ float s_red[32];
    const int lane = threadIdx.x % LANES, g = blockIdx.x * (256 / LANES) + threadIdx.x / LANES, n4 = p.group >> 2;
    const size_t row = blockIdx.y, at = static_cast<size_t>(g) * p.group;
    if (LANES == 32 && at >= static_cast<size_t>(p.n)) return;
    const float *o = p.o + row * p.n + at;
    const T *gate = static_cast<const T *>(p.gate) + row * p.ldg + at;
    float4 v[NV], z[NV];
    float ss = 0.0f;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
        const int i = lane + j * LANES;
        v[j] = z[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < n4) {
            v[j] = get4(o + 4 * i);
            z[j] = get4(gate + 4 * i);
        }
        ss += (v[j].x * v[j].x + v[j].y * v[j].y) + (v[j].z * v[j].z + v[j].w * v[j].w);
    }
    if (LANES == 32) {
#pragma unroll
        for (int s = 16; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
    } else {
        ss = dense::block_sum<256>(ss, s_red);
    }
    const float r = 1.0f / sqrtf(ss / static_cast<float>(p.group) + p.eps);
    T *out = static_cast<T *>(p.out) + row * p.ldo + at;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
        const int i = lane + j * LANES;
        if (i < n4) {
            const float4 w = __ldg(reinterpret_cast<const float4 *>(p.w) + i);
            dense::put4(out + 4 * i, make_float4(v[j].x * r * w.x * gate_of(gate, z[j].x), v[j].y * r * w.y * gate_of(gate, z[j].y), v[j].z * r * w.z * gate_of(gate, z[j].z),
                                                 v[j].w * r * w.w * gate_of(gate, z[j].w)));
        }
    }
}

constexpr size_t kRingBytes = 128 * 1024;  // two records of the largest sizes fit

template <typename T, bool DELTA>
int recur_init_kind() {
    for (void (*k)(RecurParams) : {recur_walk_kernel<T, DELTA, 1>, recur_walk_kernel<T, DELTA, 2>, recur_walk_kernel<T, DELTA, 4>})
        LBK_CUDA(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(kRingBytes)));
    return LBK_OK;
}
int recur_init(Ctx *) {
    LBK_TRY((recur_init_kind<float, true>()));
    LBK_TRY((recur_init_kind<float, false>()));
    LBK_TRY((recur_init_kind<uint16_t, true>()));
    return recur_init_kind<uint16_t, false>();
}
const InitHook kInitRecur(recur_init);

template <typename T, bool DELTA>
int launch_walk(Ctx *ctx, RecurParams &p, cudaStream_t st) {
    const size_t rec = static_cast<size_t>(p.rec) * 4;
    const size_t stages = kRingBytes / rec;
    p.stages = static_cast<int>(stages < 2 ? 2 : stages > kMaxStages ? kMaxStages : stages);
    if (p.blocks < p.stages) p.stages = p.blocks;
    // warps a block: the number that leaves the fullest SM the fewest
    int best = 1 << 30;
    for (int w = 4; w <= kMaxWarps; ++w) {
        const int blocks = (p.vdim + 4 * w - 1) / (4 * w) * p.heads, most = (blocks + ctx->sm_count - 1) / ctx->sm_count * w;
        if (most < best) {
            best = most;
            p.warps = w;
        }
    }
    void (*k)(RecurParams) = p.dp == 64 ? recur_walk_kernel<T, DELTA, 1> : p.dp == 128 ? recur_walk_kernel<T, DELTA, 2> : recur_walk_kernel<T, DELTA, 4>;
    LBK_CUDA(launch_chained(k, dim3(static_cast<unsigned>((p.vdim + 4 * p.warps - 1) / (4 * p.warps)), static_cast<unsigned>(p.heads)),
                            dim3(static_cast<unsigned>(p.warps + 1) * 32), rec * p.stages, st, p));
    LBK_CUDA(cudaGetLastError());
    ctx->launches++;
    return LBK_OK;
}

template <typename T, bool DELTA>
int launch_step(Ctx *ctx, RecurParams &p, cudaStream_t st) {
    const int x = p.a2_pitch > p.g2_pitch ? p.a2_pitch : p.g2_pitch;
    const size_t smem = (5 * static_cast<size_t>(p.dp) + 3 * static_cast<size_t>(p.vp) + static_cast<size_t>(x)) * sizeof(float);
    if (smem > 48 * 1024) return fail(LBK_ERR_UNSUPPORTED, "recurrence: the low ranks are too large");
    void (*k)(RecurParams) = p.dp == 64 ? recur_step_kernel<T, DELTA, 1> : p.dp == 128 ? recur_step_kernel<T, DELTA, 2> : recur_step_kernel<T, DELTA, 4>;
    LBK_CUDA(launch_chained(k, dim3(static_cast<unsigned>(p.heads), static_cast<unsigned>(p.n)), dim3(kStepThreads), smem, st, p));
    LBK_CUDA(cudaGetLastError());
    ctx->launches++;
    return LBK_OK;
}

template <typename T, bool DELTA>
int recur_impl(Ctx *ctx, const RecurCall &c, cudaStream_t st) {
    RecurParams p{};
    p.x = c.x;
    p.ldx = c.ldx;
    p.q_at = c.q_at;
    p.k_at = c.k_at;
    p.v_at = c.v_at;
    p.heads = static_cast<int>(c.heads);
    p.kv_heads = static_cast<int>(c.kv_heads);
    p.dim = static_cast<int>(c.dim);
    p.vdim = static_cast<int>(c.vdim);
    p.dp = static_cast<int>(recur_pitch(c.dim));
    p.vp = static_cast<int>((c.vdim + 3) / 4 * 4);
    p.rows_of_seq = c.rows_of_seq;
    p.cap = static_cast<int>(c.cap);
    p.taps = DELTA ? c.taps : 1;
    p.pos = c.pos;
    p.active = c.active;
    p.decay = c.decay;
    p.conv = c.conv;
    p.ring = c.ring;
    p.channels = static_cast<int>(2 * c.kv_heads * c.dim + c.heads * c.vdim);
    p.a = c.a;
    p.lda = c.lda;
    p.a_log = c.a_log;
    p.dt_bias = c.dt_bias;
    p.b = c.b;
    p.ldb = c.ldb;
    p.state = c.state;
    p.records = c.records;
    p.rec = ((DELTA ? 3 : 2) * kTok + 1) * p.dp + kScal + kTok * p.vp;
    p.o = c.o;
    p.err_word = ctx->err_word;
    p.total = static_cast<int>(c.rows);
    p.a_at = c.a_at;
    p.g_at = c.g_at;
    p.a2 = c.a2.w;
    p.g2 = c.g2.w;
    p.a2_pitch = static_cast<int>(c.a2.pitch);
    p.g2_pitch = static_cast<int>(c.g2.pitch);
    p.a_rank = static_cast<int>(c.a2.cols);
    p.g_rank = static_cast<int>(c.g2.cols);
    p.norm_w = c.norm_w;
    p.eps = c.eps;
    p.out = c.out;
    p.ldo = c.ldo;
    if (c.rows_of_seq < 0) {
        p.n = p.total;
        return launch_step<T, DELTA>(ctx, p, st);
    }
    for (size_t r0 = 0; r0 < c.rows; r0 += c.record_rows) {
        p.row0 = static_cast<int>(r0);
        p.n = static_cast<int>(c.rows - r0 < c.record_rows ? c.rows - r0 : c.record_rows);
        p.last = r0 + c.record_rows >= c.rows;
        p.blocks = (p.n + kTok - 1) / kTok;
        void (*k)(RecurParams) = recur_prep_kernel<T, DELTA, 1, 0>;
        if (p.dp > kPrepThreads) k = DELTA && p.taps == 4 ? recur_prep_kernel<T, DELTA, 2, 4> : recur_prep_kernel<T, DELTA, 2, 0>;
        else if (DELTA && p.taps == 4) k = recur_prep_kernel<T, DELTA, 1, 4>;
        LBK_CUDA(launch_chained(k, dim3(static_cast<unsigned>(p.heads), static_cast<unsigned>(p.blocks)), dim3(kPrepThreads), 0, st, p));
        LBK_CUDA(cudaGetLastError());
        ctx->launches++;
        LBK_TRY((launch_walk<T, DELTA>(ctx, p, st)));
    }
    return LBK_OK;
}

}  // namespace

size_t recur_pitch(size_t dim) { return dim <= 64 ? 64 : dim <= 128 ? 128 : 256; }

size_t recur_record_floats(bool delta, size_t rows, size_t heads, size_t dim, size_t vdim) {
    const size_t rec = ((delta ? 3 : 2) * kTok + 1) * recur_pitch(dim) + kScal + kTok * ((vdim + 3) / 4 * 4);
    return heads * ((rows + kTok - 1) / kTok) * rec;
}

int launch_recurrence(Ctx *ctx, const RecurCall &c, cudaStream_t st) {
    if (c.rows == 0) return LBK_OK;
    const bool batch = c.rows_of_seq < 0, low = batch && c.delta && c.a2.w && c.g2.w && c.out && c.norm_w;
    if (!c.x || !c.pos || !c.state || (!batch && !c.records) || (!c.o && !low) || (c.delta ? !c.conv || !c.ring || (!c.a && !low) || !c.a_log || !c.dt_bias || !c.b : !c.decay))
        return fail(LBK_ERR_INVALID, "recurrence: null buffer");
    if (!low && (c.a2.w || c.g2.w || c.out)) return fail(LBK_ERR_INVALID, "recurrence: low ranks and the gated norm go together, one token per sequence");
    if (!c.heads || !c.kv_heads || c.heads % c.kv_heads || !c.dim || !c.vdim || (c.delta && c.taps < 1)) return fail(LBK_ERR_SHAPE, "recurrence: inconsistent head counts or sizes");
    if (c.dim > kRecurMaxDim) return fail(LBK_ERR_UNSUPPORTED, "recurrence: key heads of at most %zu dimensions", kRecurMaxDim);
    if (c.vdim > 1024) return fail(LBK_ERR_UNSUPPORTED, "recurrence: value heads of at most 1024 dimensions");
    if (!batch && (c.record_rows == 0 || c.record_rows % kTok)) return fail(LBK_ERR_INVALID, "recurrence: records for a multiple of %d rows", kTok);
    const bool f32 = c.compute == LBK_COMPUTE_F32;
    if (c.delta) return f32 ? recur_impl<float, true>(ctx, c, st) : recur_impl<uint16_t, true>(ctx, c, st);
    return f32 ? recur_impl<float, false>(ctx, c, st) : recur_impl<uint16_t, false>(ctx, c, st);
}

int launch_gated_norm(Ctx *ctx, const GatedNormCall &c, cudaStream_t st) {
    if (c.rows == 0) return LBK_OK;
    if (!c.o || !c.w || !c.gate || !c.out || !c.group || c.n % c.group) return fail(LBK_ERR_INVALID, "gated norm: null buffer or ragged groups");
    if (c.rows > 65535) return fail(LBK_ERR_UNSUPPORTED, "at most 65535 rows per call");
    GatedParams p{c.o, c.w, c.gate, c.out, c.ldg, c.ldo, static_cast<int>(c.n), static_cast<int>(c.group), c.eps};
    const bool f32 = c.compute == LBK_COMPUTE_F32;
    const unsigned groups = static_cast<unsigned>(c.n / c.group), rows = static_cast<unsigned>(c.rows);
    const uintptr_t bits = reinterpret_cast<uintptr_t>(c.o) | reinterpret_cast<uintptr_t>(c.w) | reinterpret_cast<uintptr_t>(c.gate) | reinterpret_cast<uintptr_t>(c.out);
    if (c.group % 4 == 0 && c.ldg % 4 == 0 && c.ldo % 4 == 0 && (bits & 15) == 0 && c.group <= 8192) {
        void (*k)(GatedParams);
        const bool warp = c.group <= 256;
        if (warp) k = f32 ? gated_norm_vec_kernel<float, 32, 2> : gated_norm_vec_kernel<uint16_t, 32, 2>;
        else if (c.group <= 1024) k = f32 ? gated_norm_vec_kernel<float, 256, 1> : gated_norm_vec_kernel<uint16_t, 256, 1>;
        else if (c.group <= 4096) k = f32 ? gated_norm_vec_kernel<float, 256, 4> : gated_norm_vec_kernel<uint16_t, 256, 4>;
        else k = f32 ? gated_norm_vec_kernel<float, 256, 8> : gated_norm_vec_kernel<uint16_t, 256, 8>;
        LBK_CUDA(launch_chained(k, dim3(warp ? (groups + 7) / 8 : groups, rows), dim3(256), 0, st, p));
        LBK_CUDA(cudaGetLastError());
        ctx->launches++;
        return LBK_OK;
    }
    if (c.group <= 256) LBK_CUDA(launch_chained(f32 ? gated_norm_warp_kernel<float> : gated_norm_warp_kernel<uint16_t>, dim3((groups + 7) / 8, rows), dim3(256), 0, st, p));
    else LBK_CUDA(launch_chained(f32 ? gated_norm_block_kernel<float> : gated_norm_block_kernel<uint16_t>, dim3(groups, rows), dim3(512), 0, st, p));
    LBK_CUDA(cudaGetLastError());
    ctx->launches++;
    return LBK_OK;
}

}  // namespace lbk

using namespace lbk;

extern "C" {

size_t lbk_recurrence_state_floats(const lbk_recurrence_desc *d) { return d ? d->heads * d->vdim * recur_pitch(d->dim) : 0; }

size_t lbk_recurrence_record_floats(const lbk_recurrence_desc *d, size_t rows) {
    return d ? recur_record_floats(d->delta != 0, rows, d->heads, d->dim, d->vdim) : 0;
}

int lbk_recurrence(lbk_ctx *c, int compute, const lbk_recurrence_desc *d, const void *x_dev, size_t x_pitch, size_t rows, int rows_of_seq,
                   const int32_t *pos_dev, const int32_t *active_dev, size_t cap, const float *decay_dev, const float *conv_dev, void *ring_dev,
                   const float *a_dev, const float *a_log_dev, const float *dt_bias_dev, const float *b_dev, float *state_dev, float *records_dev,
                   size_t record_rows, float *o_dev, void *stream) {
    if (!c || !d) return fail(LBK_ERR_INVALID, "lbk_recurrence: null argument");
    Ctx *ctx = reinterpret_cast<Ctx *>(c);
    LBK_CUDA(cudaSetDevice(ctx->device));
    RecurCall r;
    r.compute = compute;
    r.delta = d->delta != 0;
    r.heads = d->heads;
    r.kv_heads = d->kv_heads;
    r.dim = d->dim;
    r.vdim = d->vdim;
    r.taps = static_cast<int>(d->taps);
    r.x = x_dev;
    r.ldx = static_cast<long>(x_pitch);
    r.k_at = static_cast<int>(d->kv_heads * d->dim);
    r.v_at = 2 * r.k_at;
    r.rows = rows;
    r.rows_of_seq = rows_of_seq;
    r.pos = pos_dev;
    r.active = active_dev;
    r.cap = cap;
    r.decay = decay_dev;
    r.conv = conv_dev;
    r.ring = ring_dev;
    r.a = a_dev;
    r.lda = static_cast<long>(d->heads * d->dim);
    r.a_log = a_log_dev;
    r.dt_bias = dt_bias_dev;
    r.b = b_dev;
    r.ldb = static_cast<long>(d->heads);
    r.state = state_dev;
    r.records = records_dev;
    r.record_rows = record_rows;
    r.o = o_dev;
    return launch_recurrence(ctx, r, static_cast<cudaStream_t>(stream));
}

int lbk_gated_norm(lbk_ctx *c, int compute, const float *o_dev, size_t rows, size_t n, size_t group, const float *w_dev, const void *gate_dev,
                   size_t gate_pitch, float eps, void *out_dev, size_t out_pitch, void *stream) {
    if (!c) return fail(LBK_ERR_INVALID, "lbk_gated_norm: context is null");
    Ctx *ctx = reinterpret_cast<Ctx *>(c);
    LBK_CUDA(cudaSetDevice(ctx->device));
    GatedNormCall g;
    g.compute = compute;
    g.o = o_dev;
    g.rows = rows;
    g.n = n;
    g.group = group;
    g.w = w_dev;
    g.gate = gate_dev;
    g.ldg = static_cast<long>(gate_pitch);
    g.eps = eps;
    g.out = out_dev;
    g.ldo = static_cast<long>(out_pitch);
    return launch_gated_norm(ctx, g, static_cast<cudaStream_t>(stream));
}

}  // extern "C"
