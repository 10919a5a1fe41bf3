// Linear recurrences: attention whose past is a matrix S [dim x vdim] per head instead of a list of keys.
//
//   plain   S <- decay S + k v^T;  o = S^T q                     (decay: a constant of the head)
//   delta   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q      (g: per token, head and key channel)
//
// The state and everything that enters it are f32 on the FMA pipes; nothing of a recurrence is rounded to 16 bits. Tokens
// are taken four at a time. With S the state in front of four tokens, G_i the product of their decays up to and including
// token i, and "after j" the product of those behind token j:
//
//   a_i = S^T (k_i G_i)      b_i = S^T (q_i G_i)
//   u_i = beta_i (v_i - a_i - sum_{j<i} c_ij u_j)       c_ij = k_i . (k_j x decays j+1 .. i)       (plain: u_i = v_i)
//   o_i = b_i + sum_{j<=i} p_ij u_j                     p_ij = q_i . (k_j x decays j+1 .. i)
//   S  <- G_3 S + sum_j (k_j x decays after j) u_j^T
//
// which is the recurrence itself, reordered: one multiplication of the state by decays instead of four and products of
// at most four decays (never a quotient, so strong decays underflow to zero as they should). Kernels:
//
//   recur_prep_kernel   one block per (four tokens, head): silu(q, k, v) or, for delta, short convolution + silu, unit
//                       vectors, decays and step sizes; writes one record per (four tokens, head) with the vectors
//                       and numbers above. Every token block is independent of every other.
//   recur_kernel        one block per (sequence, head, slice of value columns) walks the records in order. A column of S
//                       lives in the registers of eight lanes (dim / 8 values each, as packed pairs for the two-wide
//                       FMA), a warp holds 4 or 8 columns. A producer lane brings the records into a ring of shared
//                       memory with bulk copies; the dots over eight lanes meet by transposing shuffles.
//   gated_norm_kernel   the read-out divided by its root mean square per group, times a weight and sigmoid(gate).
//
// A sequence at position 0 starts from a zero state whatever the buffer holds, so a slot that is used again needs no
// clearing. Convolution inputs that later tokens need stay in a ring by position; recur_kernel stores them (after every
// prep block of the pass has read the old ones).
#include "lbk_dense_dev.cuh"
#include "lbk_mixers.cuh"
#include "lbk_ptx.cuh"

namespace lbk {

namespace {

constexpr int kTok = 4;             // tokens per record
constexpr int kPrepThreads = 128;
constexpr int kScal = 32;           // numbers of a record: c 0..5, beta 8..11, p 12 + 4 i + j
constexpr int kWarps = 4;           // warps that hold columns
constexpr uint32_t kWaitLimit = 1u << 22;

struct RecurParams {
    const void *x;
    long ldx;
    int q_at, k_at, v_at, heads, kv_heads, dim, vdim, dp, vp;
    int n, rows_of_seq, row0, blocks, cap, taps, last, total;
    const int *pos, *active;
    const float *decay;
    const float *conv;
    void *ring;
    int channels;
    const float *a;
    long lda;
    const float *a_log, *dt_bias, *b;
    long ldb;
    float *state, *records;
    int rec;                        // floats of a record
    float *o;
    int stages;
    int *err_word;
};

__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }

// Sums of N values over the 128 threads of a prep block; every thread gets all of them.
template <int N>
__device__ __forceinline__ void prep_sum(float (&v)[N], float *s_red) {
#pragma unroll
    for (int i = 0; i < N; ++i)
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) v[i] += __shfl_xor_sync(0xffffffffu, v[i], o);
    __syncthreads();
    if ((threadIdx.x & 31) == 0)
#pragma unroll
        for (int i = 0; i < N; ++i) s_red[(threadIdx.x >> 5) * N + i] = v[i];
    __syncthreads();
#pragma unroll
    for (int i = 0; i < N; ++i) v[i] = (s_red[i] + s_red[N + i]) + (s_red[2 * N + i] + s_red[3 * N + i]);
}

// NB: dimensions a thread takes (dp / 128, at least 1)
template <typename T, bool DELTA, int NB>
__global__ void __launch_bounds__(kPrepThreads) recur_prep_kernel(const RecurParams p) {
    ptx::pdl_trigger();
    ptx::pdl_wait();
    __shared__ float s_red[4 * 16];
    const int h = blockIdx.x, blk = blockIdx.y, tid = threadIdx.x;
    const bool batch = p.rows_of_seq < 0;
    const int seq = batch ? blk : p.rows_of_seq;
    const int row0 = batch ? blk : p.row0 + blk * kTok;    // row of token 0 of this record
    const int cnt = batch ? 1 : min(kTok, p.row0 + p.n - row0);
    const int pos0 = batch ? p.pos[blk] : p.pos[0];        // position of row `batch ? blk : 0`
    if (pos0 < 0 || pos0 + (batch ? 1 : p.total) > p.cap) {
        if (tid == 0) atomicExch(p.err_word, 7);
        return;
    }
    const T *x = static_cast<const T *>(p.x);
    float *rec = p.records + (static_cast<size_t>(batch ? blk * p.heads + h : h * p.blocks + blk)) * p.rec;
    const int kvh = h / (p.heads / p.kv_heads);
    // the value of channel `ch` for token i, silu'd (and convolved)
    auto value = [&](int at, int ch, int i) -> float {
        const T *col = x + at + ch;
        if (!DELTA) return dense::get(col + static_cast<size_t>(row0 + i) * p.ldx);
        const int cc = at - p.q_at + ch;
        const float *w = p.conv + static_cast<size_t>(cc) * p.taps;
        float y = 0.0f;
        for (int j = 0; j < p.taps; ++j) {
            const int back = p.taps - 1 - j;
            const int r = batch ? -back : row0 + i - back;  // row, or how far in front of this pass
            float v = 0.0f;
            if (back == 0 || (!batch && r >= 0)) {
                v = dense::get(col + static_cast<size_t>(batch ? row0 : r) * p.ldx);
            } else if (pos0 + r >= 0) {
                v = dense::get(static_cast<const T *>(p.ring) + (static_cast<size_t>(seq) * p.taps + (pos0 + r) % p.taps) * p.channels + cc);
            }
            y = fmaf(v, w[j], y);
        }
        return dense::silu<true>(y);
    };
    float q[NB][kTok], k[NB][kTok], g[NB][kTok];
#pragma unroll
    for (int b = 0; b < NB; ++b) {
        const int d = tid + b * kPrepThreads;
#pragma unroll
        for (int i = 0; i < kTok; ++i) {
            const bool live = d < p.dim && i < cnt;
            q[b][i] = live ? value(p.q_at, kvh * p.dim + d, i) : 0.0f;
            k[b][i] = live ? value(p.k_at, kvh * p.dim + d, i) : 0.0f;
            g[b][i] = 1.0f;
        }
    }
    if (DELTA) {
        float ss[2 * kTok] = {};
#pragma unroll
        for (int b = 0; b < NB; ++b)
#pragma unroll
            for (int i = 0; i < kTok; ++i) {
                ss[i] = fmaf(q[b][i], q[b][i], ss[i]);
                ss[kTok + i] = fmaf(k[b][i], k[b][i], ss[kTok + i]);
            }
        prep_sum(ss, s_red);
        const float qs = 1.0f / sqrtf(static_cast<float>(p.dim));
        const float rate = expf(p.a_log[h]);
#pragma unroll
        for (int b = 0; b < NB; ++b) {
            const int d = tid + b * kPrepThreads;
#pragma unroll
            for (int i = 0; i < kTok; ++i) {
                q[b][i] *= qs / sqrtf(ss[i] + 1e-6f);
                k[b][i] *= 1.0f / sqrtf(ss[kTok + i] + 1e-6f);
                if (d < p.dim && i < cnt)
                    g[b][i] = expf(-rate * softplus(p.a[static_cast<size_t>(row0 + i) * p.lda + h * p.dim + d] + p.dt_bias[h * p.dim + d]));
            }
        }
    } else {
        const float decay = p.decay[h];
#pragma unroll
        for (int b = 0; b < NB; ++b)
#pragma unroll
            for (int i = 0; i < kTok; ++i) g[b][i] = i < cnt ? decay : 1.0f;
    }
    // the record
    float *rk = rec, *rq = rec + (DELTA ? kTok : 0) * p.dp, *rh = rq + kTok * p.dp, *rg = rh + kTok * p.dp, *rs = rg + p.dp, *rv = rs + kScal;
    float dots[16] = {};                                   // p (10), c (6)
#pragma unroll
    for (int b = 0; b < NB; ++b) {
        const int d = tid + b * kPrepThreads;
        float after = 1.0f, upto = 1.0f;
#pragma unroll
        for (int i = 0; i < kTok; ++i) {
            upto *= g[b][i];
            if (d < p.dp) {
                if (DELTA) rk[i * p.dp + d] = k[b][i] * upto;
                rq[i * p.dp + d] = q[b][i] * upto;
            }
        }
        if (d < p.dp) rg[d] = upto;
#pragma unroll
        for (int j = kTok - 1; j >= 0; --j) {
            if (d < p.dp) rh[j * p.dp + d] = k[b][j] * after;
            after *= g[b][j];
        }
        int at = 0, ac = 10;
#pragma unroll
        for (int i = 0; i < kTok; ++i) {
            float f = 1.0f;
#pragma unroll
            for (int j = i; j >= 0; --j) {                 // p_ij at i (i + 1) / 2 + j, c_ij at 10 + i (i - 1) / 2 + j
                dots[at + j] = fmaf(q[b][i] * f, k[b][j], dots[at + j]);
                if (DELTA && j < i) dots[ac + j] = fmaf(k[b][i] * f, k[b][j], dots[ac + j]);
                f *= g[b][j];
            }
            at += i + 1;
            ac += i;
        }
    }
    __syncthreads();
    prep_sum(dots, s_red);
    if (tid < kScal) {
        float v = 0.0f;
        if (tid < 6) {
#pragma unroll
            for (int e = 0; e < 6; ++e)
                if (e == tid) v = dots[10 + e];
        } else if (tid >= 8 && tid < 12) {
            if (DELTA && tid - 8 < cnt) v = dense::sigmoid(p.b[static_cast<size_t>(row0 + tid - 8) * p.ldb + h]);
        } else if (tid >= 12 && tid < 28) {
            const int i = (tid - 12) >> 2, j = (tid - 12) & 3;
            if (j <= i) {
#pragma unroll
                for (int e = 0; e < 10; ++e)
                    if (e == i * (i + 1) / 2 + j) v = dots[e];
            }
        }
        rs[tid] = v;
    }
    for (int e = tid; e < kTok * p.vp; e += kPrepThreads) {
        const int i = e / p.vp, c = e - i * p.vp;
        rv[e] = i < cnt && c < p.vdim ? value(p.v_at, h * p.vdim + c, i) : 0.0f;
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

// J: 16-byte units of a column per lane (dp = 32 J); NC: columns per group of eight lanes
template <typename T, bool DELTA, int J, int NC>
__global__ void __launch_bounds__((kWarps + 1) * 32) recur_kernel(const RecurParams p) {
    extern __shared__ __align__(16) uint8_t rc_smem[];
    __shared__ __align__(8) uint64_t s_bar[32];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int h = blockIdx.y, slice = blockIdx.x;
    const bool batch = p.rows_of_seq < 0;
    const int seq = batch ? blockIdx.z : p.rows_of_seq;
    const uint32_t bar0 = ptx::smem_u32(s_bar), ring0 = ptx::smem_u32(rc_smem);
    const uint32_t bytes = static_cast<uint32_t>(p.rec) * 4;
    if (tid == 0) {
        for (int s = 0; s < p.stages; ++s) {
            ptx::mbar_init(bar0 + s * 8, 1);
            ptx::mbar_init(bar0 + (16 + s) * 8, kWarps);
        }
        ptx::fence_barrier_init();
    }
    __syncthreads();
    ptx::pdl_trigger();
    ptx::pdl_wait();
    const int pos_first = batch ? p.pos[seq] : p.pos[0];
    const bool fits = pos_first >= 0 && pos_first + (batch ? 1 : p.total) <= p.cap;   // the prep kernel has flagged it
    const bool keep = !batch || !p.active || p.active[seq] != 0;
    const int blocks = fits ? p.blocks : 0;
    if (warp == kWarps) {
        if (lane == 0) {
            const float *rec = p.records + static_cast<size_t>(batch ? seq * p.heads + h : h * p.blocks) * p.rec;
            for (int b = 0; b < blocks; ++b) {
                const int s = b % p.stages, round = b / p.stages;
                if (round > 0 && !ptx::mbar_wait(bar0 + (16 + s) * 8, (round - 1) & 1, kWaitLimit)) {
                    atomicExch(p.err_word, 5);
                    break;
                }
                ptx::mbar_arrive_expect_tx(bar0 + s * 8, bytes);
                bulk_load(ring0 + s * bytes, rec + static_cast<size_t>(b) * p.rec, bytes, bar0 + s * 8);
            }
        }
    } else {
        const int l = lane & 7, cg = lane >> 3;
        const int col0 = (slice * kWarps + warp) * 4 * NC + cg * NC;
        const int pos0 = pos_first + (batch ? 0 : p.row0);
        float *st = p.state + static_cast<size_t>(seq * p.heads + h) * p.vdim * p.dp;
        u64 S[NC][J][2];
#pragma unroll
        for (int c = 0; c < NC; ++c)
#pragma unroll
            for (int j = 0; j < J; ++j) {
                ulonglong2 v = make_ulonglong2(0, 0);
                if (pos0 > 0 && col0 + c < p.vdim) v = *reinterpret_cast<const ulonglong2 *>(st + static_cast<size_t>(col0 + c) * p.dp + 4 * (l + 8 * j));
                S[c][j][0] = v.x;
                S[c][j][1] = v.y;
            }
        bool ok = true;
        int s = 0, phase = 0;
        for (int b = 0; b < blocks; ++b) {
            if (!__all_sync(0xffffffffu, ptx::mbar_wait(bar0 + s * 8, phase, kWaitLimit))) {
                ok = false;
                break;
            }
            const float *rec = reinterpret_cast<const float *>(rc_smem + static_cast<size_t>(s) * bytes);
            const float *rk = rec, *rq = rec + (DELTA ? kTok : 0) * p.dp, *rh = rq + kTok * p.dp, *rg = rh + kTok * p.dp, *rs = rg + p.dp, *rv = rs + kScal;
            u64 a[NC][kTok], o[NC][kTok];
#pragma unroll
            for (int c = 0; c < NC; ++c)
#pragma unroll
                for (int i = 0; i < kTok; ++i) a[c][i] = o[c][i] = 0;
#pragma unroll
            for (int j = 0; j < J; ++j) {
                const int off = 4 * (l + 8 * j);
#pragma unroll
                for (int i = 0; i < kTok; ++i) {
                    if (DELTA) {
                        const ulonglong2 v = *reinterpret_cast<const ulonglong2 *>(rk + i * 32 * J + off);
#pragma unroll
                        for (int c = 0; c < NC; ++c) a[c][i] = fma2(v.y, S[c][j][1], fma2(v.x, S[c][j][0], a[c][i]));
                    }
                    const ulonglong2 w = *reinterpret_cast<const ulonglong2 *>(rq + i * 32 * J + off);
#pragma unroll
                    for (int c = 0; c < NC; ++c) o[c][i] = fma2(w.y, S[c][j][1], fma2(w.x, S[c][j][0], o[c][i]));
                }
            }
            float u[NC][kTok], mine[NC];  // mine: b_i of token i = l & 3
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                float r[kTok];
                if (DELTA) {             // lanes 0..3 end up with a_0 .. a_3, lanes 4..7 with b_0 .. b_3
                    const bool up = (l & 4) != 0;
#pragma unroll
                    for (int i = 0; i < kTok; ++i) {
                        const float va = sum2(a[c][i]), vb = sum2(o[c][i]);
                        r[i] = (up ? vb : va) + __shfl_xor_sync(0xffffffffu, up ? va : vb, 4);
                    }
                } else {
#pragma unroll
                    for (int i = 0; i < kTok; ++i) {
                        const float vb = sum2(o[c][i]);
                        r[i] = vb + __shfl_xor_sync(0xffffffffu, vb, 4);
                    }
                }
                const bool b2 = (l & 2) != 0, b1 = (l & 1) != 0;
                const float r0 = (b2 ? r[2] : r[0]) + __shfl_xor_sync(0xffffffffu, b2 ? r[0] : r[2], 2);
                const float r1 = (b2 ? r[3] : r[1]) + __shfl_xor_sync(0xffffffffu, b2 ? r[1] : r[3], 2);
                mine[c] = (b1 ? r1 : r0) + __shfl_xor_sync(0xffffffffu, b1 ? r0 : r1, 1);
                const float *vc = rv + min(col0 + c, p.vdim - 1);
#pragma unroll
                for (int i = 0; i < kTok; ++i) u[c][i] = vc[i * p.vp];
                if (DELTA) {
                    const float4 beta = *reinterpret_cast<const float4 *>(rs + 8), c0 = *reinterpret_cast<const float4 *>(rs);
                    const float2 c1 = *reinterpret_cast<const float2 *>(rs + 4);
                    float t[kTok];
#pragma unroll
                    for (int i = 0; i < kTok; ++i) t[i] = u[c][i] - __shfl_sync(0xffffffffu, mine[c], (lane & 24) | i);
                    u[c][0] = beta.x * t[0];
                    u[c][1] = beta.y * (t[1] - c0.x * u[c][0]);
                    u[c][2] = beta.z * (t[2] - c0.y * u[c][0] - c0.z * u[c][1]);
                    u[c][3] = beta.w * (t[3] - c0.w * u[c][0] - c1.x * u[c][1] - c1.y * u[c][2]);
                }
            }
            if (l >= 4) {
                const int i = l & 3, t = batch ? seq : p.row0 + b * kTok + i;
                const float4 pr = *reinterpret_cast<const float4 *>(rs + 12 + 4 * i);
                if (batch ? i == 0 : b * kTok + i < p.n) {
#pragma unroll
                    for (int c = 0; c < NC; ++c)
                        if (col0 + c < p.vdim)
                            p.o[(static_cast<size_t>(t) * p.heads + h) * p.vdim + col0 + c] =
                                mine[c] + ((pr.x * u[c][0] + pr.y * u[c][1]) + (pr.z * u[c][2] + pr.w * u[c][3]));
                }
            }
            u64 uu[NC][kTok];
#pragma unroll
            for (int c = 0; c < NC; ++c)
#pragma unroll
                for (int i = 0; i < kTok; ++i) uu[c][i] = pack2(u[c][i], u[c][i]);
#pragma unroll
            for (int j = 0; j < J; ++j) {
                const int off = 4 * (l + 8 * j);
                const ulonglong2 g = *reinterpret_cast<const ulonglong2 *>(rg + off);
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    S[c][j][0] = mul2(g.x, S[c][j][0]);
                    S[c][j][1] = mul2(g.y, S[c][j][1]);
                }
#pragma unroll
                for (int i = 0; i < kTok; ++i) {
                    const ulonglong2 v = *reinterpret_cast<const ulonglong2 *>(rh + i * 32 * J + off);
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        S[c][j][0] = fma2(v.x, uu[c][i], S[c][j][0]);
                        S[c][j][1] = fma2(v.y, uu[c][i], S[c][j][1]);
                    }
                }
            }
            __syncwarp();
            if (lane == 0) ptx::mbar_arrive(bar0 + (16 + s) * 8);
            if (++s == p.stages) {
                s = 0;
                phase ^= 1;
            }
        }
        if (!ok && lane == 0) atomicExch(p.err_word, 5);
        if (ok && fits && keep) {
#pragma unroll
            for (int c = 0; c < NC; ++c)
                if (col0 + c < p.vdim)
#pragma unroll
                    for (int j = 0; j < J; ++j)
                        *reinterpret_cast<ulonglong2 *>(st + static_cast<size_t>(col0 + c) * p.dp + 4 * (l + 8 * j)) = make_ulonglong2(S[c][j][0], S[c][j][1]);
            if (DELTA && slice == 0 && p.last && p.taps > 1) {
                // the inputs later tokens will convolve with: the last taps - 1 of this pass, this head's channels
                const T *x = static_cast<const T *>(p.x);
                const int group = p.heads / p.kv_heads, qk = h % group == 0 ? 2 * p.dim : 0, all = qk + p.vdim;
                const int rows = batch ? 1 : min(p.taps - 1, p.total);
                for (int e = tid; e < rows * all; e += kWarps * 32) {
                    const int r = e / all, c = e - r * all;
                    const int col = c < qk ? (c < p.dim ? p.q_at : p.k_at - p.dim) + (h / group) * p.dim + c : p.v_at + h * p.vdim + c - qk;
                    const int row = batch ? seq : p.total - rows + r, ps = pos_first + (batch ? 0 : row);
                    static_cast<T *>(p.ring)[(static_cast<size_t>(seq) * p.taps + ps % p.taps) * p.channels + col - p.q_at] = x[static_cast<size_t>(row) * p.ldx + col];
                }
            }
        }
    }
    __syncthreads();
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

constexpr size_t kRingBytes = 96 * 1024;  // two records of the largest sizes fit

template <typename T, bool DELTA>
int recur_init_kind() {
    for (void (*k)(RecurParams) : {recur_kernel<T, DELTA, 1, 1>, recur_kernel<T, DELTA, 1, 2>, recur_kernel<T, DELTA, 2, 1>, recur_kernel<T, DELTA, 2, 2>,
                                   recur_kernel<T, DELTA, 4, 1>, recur_kernel<T, DELTA, 4, 2>, recur_kernel<T, DELTA, 8, 1>, recur_kernel<T, DELTA, 8, 2>})
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

template <typename T, bool DELTA, int J>
int launch_walk(Ctx *ctx, RecurParams &p, cudaStream_t st) {
    const size_t rec = static_cast<size_t>(p.rec) * 4;
    size_t stages = kRingBytes / rec;
    p.stages = static_cast<int>(stages < 2 ? 2 : stages > 12 ? 12 : stages);
    if (p.blocks < p.stages) p.stages = p.blocks;
    const unsigned seqs = p.rows_of_seq < 0 ? static_cast<unsigned>(p.n) : 1u;
    // eight columns a warp halve the reads of shared memory, four spread a few heads over more SMs
    const size_t wide = (static_cast<size_t>(p.vdim) + 31) / 32 * p.heads * seqs;
    const bool two = wide >= 100;
    const unsigned slices = static_cast<unsigned>((p.vdim + (two ? 31 : 15)) / (two ? 32 : 16));
    void (*k)(RecurParams) = two ? recur_kernel<T, DELTA, J, 2> : recur_kernel<T, DELTA, J, 1>;
    const size_t smem = rec * p.stages;
    LBK_CUDA(launch_chained(k, dim3(slices, static_cast<unsigned>(p.heads), seqs), dim3((kWarps + 1) * 32), smem, st, p));
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
    const size_t run = c.rows_of_seq < 0 ? c.rows : c.record_rows;
    for (size_t r0 = 0; r0 < c.rows; r0 += run) {
        p.row0 = static_cast<int>(r0);
        p.n = static_cast<int>(c.rows - r0 < run ? c.rows - r0 : run);
        p.last = r0 + run >= c.rows;
        p.blocks = c.rows_of_seq < 0 ? 1 : (p.n + kTok - 1) / kTok;
        const dim3 grid(static_cast<unsigned>(p.heads), static_cast<unsigned>(c.rows_of_seq < 0 ? p.n : p.blocks));
        LBK_CUDA(launch_chained(p.dp > kPrepThreads ? recur_prep_kernel<T, DELTA, 2> : recur_prep_kernel<T, DELTA, 1>, grid, dim3(kPrepThreads), 0, st, p));
        LBK_CUDA(cudaGetLastError());
        ctx->launches++;
        switch (p.dp) {
            case 32: LBK_TRY((launch_walk<T, DELTA, 1>(ctx, p, st))); break;
            case 64: LBK_TRY((launch_walk<T, DELTA, 2>(ctx, p, st))); break;
            case 128: LBK_TRY((launch_walk<T, DELTA, 4>(ctx, p, st))); break;
            default: LBK_TRY((launch_walk<T, DELTA, 8>(ctx, p, st))); break;
        }
    }
    return LBK_OK;
}

}  // namespace

size_t recur_pitch(size_t dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 128 ? 128 : 256; }

size_t recur_record_floats(bool delta, size_t rows, bool batch, size_t heads, size_t dim, size_t vdim) {
    const size_t rec = ((delta ? 3 : 2) * kTok + 1) * recur_pitch(dim) + kScal + kTok * ((vdim + 3) / 4 * 4);
    return heads * (batch ? rows : (rows + kTok - 1) / kTok) * rec;
}

int launch_recurrence(Ctx *ctx, const RecurCall &c, cudaStream_t st) {
    if (c.rows == 0) return LBK_OK;
    if (!c.x || !c.pos || !c.state || !c.records || !c.o || (c.delta ? !c.conv || !c.ring || !c.a || !c.a_log || !c.dt_bias || !c.b : !c.decay))
        return fail(LBK_ERR_INVALID, "recurrence: null buffer");
    if (!c.heads || !c.kv_heads || c.heads % c.kv_heads || !c.dim || !c.vdim || (c.delta && c.taps < 1)) return fail(LBK_ERR_SHAPE, "recurrence: inconsistent head counts or sizes");
    if (c.dim > kRecurMaxDim) return fail(LBK_ERR_UNSUPPORTED, "recurrence: key heads of at most %zu dimensions", kRecurMaxDim);
    if (c.vdim > 1024) return fail(LBK_ERR_UNSUPPORTED, "recurrence: value heads of at most 1024 dimensions");
    if (c.rows_of_seq >= 0 && (c.record_rows == 0 || c.record_rows % kTok)) return fail(LBK_ERR_INVALID, "recurrence: records for a multiple of %d rows", kTok);
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
    if (c.group <= 256) LBK_CUDA(launch_chained(f32 ? gated_norm_warp_kernel<float> : gated_norm_warp_kernel<uint16_t>, dim3((groups + 7) / 8, rows), dim3(256), 0, st, p));
    else LBK_CUDA(launch_chained(f32 ? gated_norm_block_kernel<float> : gated_norm_block_kernel<uint16_t>, dim3(groups, rows), dim3(512), 0, st, p));
    LBK_CUDA(cudaGetLastError());
    ctx->launches++;
    return LBK_OK;
}

}  // namespace lbk
