// Latent attention: a position caches one vector c (kv_rank values, normed) and one rotated key part shared by all heads,
// instead of keys and values per head. Head h's key is [W_uk,h c ; k_rot], its value W_uv,h c.
//
// Two forms of the same attention:
//
//   absorbing   (W_uk,h^T q) . c + q_rot . k_rot is the score, W_uv,h (sum of p c) the output: all heads read the same
//               rows, [c | k_rot] as keys and c as values, so the cache is read once for all of them. Decode, short
//               portions, and everything in 32-bit.
//   expanding   keys and values of all positions are written out per head by one projection of the cached latents, and
//               prompt rows go to the tcgen05 attention (lbk_attn_tc.cu). Fewer operations a row, more a position.
//
// A cache row is [c, zeros to kvp | k_rot, zeros], the pitch a multiple of 64 values, so that it is the operand of a
// projection as it lies there. Kernels:
//
//   latent_prep_kernel    a token's projections: norm of the query latent; norm of c and rotation of the key part, stored
//                         into the cache. Angles: position * frequency in double, reduced to one turn, then sincospif.
//   latent_rotate_kernel  rotated parts of all heads of the queries in place (expanding form)
//   latent_absorb_kernel, latent_absorb_mma_kernel  W_uk,h^T q and the rotated part: a query against cache rows (32-bit, bf16)
//   latent_attn_kernel    bf16, tcgen05: 64 positions' rows come by TMA and serve both products as they lie there. The
//                         scores are taken transposed, positions x heads (the rows are the MMA's M side, 16 or 32 heads
//                         its N side, so few heads cost little), and so is the output, latent dimensions x heads: the
//                         rows again, now as the MN-major operand, times the probabilities (two bf16 terms side by side
//                         on the N side). Both accumulate in tensor memory; the running maxima move lazily as in
//                         lbk_attn_tc.cu. Two buffers of rows: one is filled while the other is worked on. Slices of the
//                         positions over the blocks of the grid.
//   latent_merge_kernel   bf16: merges the slices of up to 8 rows and multiplies by W_uv,h on mma.sync; the head's gate
//   latent_out_kernel     32-bit: W_uv,h and the gate
#include <algorithm>
#include <cmath>

#include "lbk_dense_dev.cuh"
#include "lbk_mixers.cuh"
#include "lbk_ptx.cuh"
#include "lbk_tcgen05.cuh"

namespace lbk {

namespace {

struct Angles {
    const double *freq;
    int dims;
    float factor;
};
// (cos, sin) of pair i at position pos
__device__ __forceinline__ float2 turn(const Angles &r, int i, int pos) {
    constexpr double kPerTurn = 0.15915494309189533576888376337251;  // 1 / (2 pi)
    const double a = static_cast<double>(pos) * r.freq[i] * kPerTurn;
    float s, c;
    sincospif(2.0f * static_cast<float>(a - floor(a)), &s, &c);
    return make_float2(c * r.factor, s * r.factor);
}
Angles angles(const Rotation &r) { return Angles{r.freq, r.dims, r.factor}; }

struct PrepParams {
    const float *z;
    long ldz, ldq;
    int q_rank, kv_rank, rot_dim, kvp, pitch, rows, rows_of_seq, cap;
    const int *pos;
    const float *q_norm, *kv_norm;
    float eps;
    Angles rot;
    void *cq, *cache;
    int *err_word;
};

template <typename T>
__global__ void __launch_bounds__(256) latent_prep_kernel(const PrepParams p) {
    ptx::pdl_trigger();
    ptx::pdl_wait();
    __shared__ float2 s_red[8];
    const int row = blockIdx.x, tid = threadIdx.x;
    const float *z = p.z + static_cast<size_t>(row) * p.ldz, *kv = z + p.q_rank;
    constexpr int kHeld = 8;                               // the first values of a thread stay in registers
    float held[kHeld];
    float sq = 0.0f, sk = 0.0f;
#pragma unroll
    for (int j = 0; j < kHeld; ++j) {
        const int i = tid + 256 * j;
        held[j] = i < p.q_rank ? z[i] : 0.0f;
        sq = fmaf(held[j], held[j], sq);
    }
    for (int i = tid + 256 * kHeld; i < p.q_rank; i += 256) sq = fmaf(z[i], z[i], sq);
    if (p.cache)
        for (int i = tid; i < p.kv_rank; i += 256) sk = fmaf(kv[i], kv[i], sk);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        sq += __shfl_xor_sync(0xffffffffu, sq, o);
        sk += __shfl_xor_sync(0xffffffffu, sk, o);
    }
    if ((tid & 31) == 0) s_red[tid >> 5] = make_float2(sq, sk);
    __syncthreads();
    sq = sk = 0.0f;
#pragma unroll
    for (int w = 0; w < 8; ++w) {
        sq += s_red[w].x;
        sk += s_red[w].y;
    }
    const float rq = 1.0f / sqrtf(sq / static_cast<float>(p.q_rank) + p.eps);
    T *cq = static_cast<T *>(p.cq) + static_cast<size_t>(row) * p.ldq;
#pragma unroll
    for (int j = 0; j < kHeld; ++j) {
        const int i = tid + 256 * j;
        if (i < p.q_rank) dense::put(cq + i, held[j] * rq * p.q_norm[i]);
    }
    for (int i = tid + 256 * kHeld; i < p.q_rank; i += 256) dense::put(cq + i, z[i] * rq * p.q_norm[i]);
    if (!p.cache) return;
    const int seq = p.rows_of_seq >= 0 ? p.rows_of_seq : row, pos = p.rows_of_seq >= 0 ? p.pos[0] + row : p.pos[row];
    if (pos < 0 || pos >= p.cap) {
        if (tid == 0) atomicExch(p.err_word, 7);
        return;
    }
    const float rk = 1.0f / sqrtf(sk / static_cast<float>(p.kv_rank) + p.eps);
    T *dst = static_cast<T *>(p.cache) + (static_cast<size_t>(seq) * p.cap + pos) * p.pitch;
    for (int i = tid; i < p.kv_rank; i += 256) dense::put(dst + i, kv[i] * rk * p.kv_norm[i]);
    for (int i = tid; i < p.rot_dim / 2; i += 256) {
        const float2 cs = turn(p.rot, i, pos);
        const float u = kv[p.kv_rank + 2 * i], v = kv[p.kv_rank + 2 * i + 1];
        dense::put(dst + p.kvp + 2 * i, u * cs.x - v * cs.y);
        dense::put(dst + p.kvp + 2 * i + 1, v * cs.x + u * cs.y);
    }
}

struct QueryParams {
    void *q, *ql;
    int rows, rows_of_seq, heads, dim, dp, rot_dim, rp, kv_rank, kvp, pitch;
    const int *pos;
    Angles rot;
    const uint16_t *uk;
    int uk_pitch;
};

// queries [rows][heads][dp + rp]: the rotated part turned in place, zeros in the padding
template <typename T>
__global__ void __launch_bounds__(256) latent_rotate_kernel(const QueryParams p) {
    ptx::pdl_trigger();
    ptx::pdl_wait();
    extern __shared__ float2 s_turn[];
    const int row = blockIdx.x, tid = threadIdx.x, half = p.rot_dim / 2;
    const int pos = p.rows_of_seq >= 0 ? p.pos[0] + row : p.pos[row];
    for (int i = tid; i < half; i += 256) s_turn[i] = turn(p.rot, i, pos);
    __syncthreads();
    T *q = static_cast<T *>(p.q) + static_cast<size_t>(row) * p.heads * (p.dp + p.rp);
    for (int e = tid; e < p.heads * half; e += 256) {
        const int h = e / half, i = e - h * half;
        T *d = q + static_cast<size_t>(h) * (p.dp + p.rp) + p.dp + 2 * i;
        const float u = dense::get(d), v = dense::get(d + 1);
        dense::put(d, u * s_turn[i].x - v * s_turn[i].y);
        dense::put(d + 1, v * s_turn[i].x + u * s_turn[i].y);
    }
    const int pd = p.dp - p.dim, pr = p.rp - p.rot_dim;
    if (pd + pr)
        for (int e = tid; e < p.heads * (pd + pr); e += 256) {
            const int h = e / (pd + pr), i = e - h * (pd + pr);
            dense::put(q + static_cast<size_t>(h) * (p.dp + p.rp) + (i < pd ? p.dim + i : p.dp + p.rot_dim + i - pd), 0.0f);
        }
}

// 32-bit. One block: head blockIdx.x, 128 latent dimensions, four tokens. Threads: 16 groups of 8 dimensions x 16 shares of the
// head's unrotated dimensions.
constexpr int kAbsCols = 128, kAbsTok = 4;
__global__ void __launch_bounds__(256) latent_absorb_kernel(const QueryParams p) {
    using T = float;
    extern __shared__ float s_q[];                       // [kAbsTok][dim]
    __shared__ float s_part[8][kAbsTok][kAbsCols];
    const int h = blockIdx.x, c0 = blockIdx.y * kAbsCols, t0 = blockIdx.z * kAbsTok, tid = threadIdx.x;
    ptx::pdl_trigger();
    ptx::pdl_wait();
    const int toks = min(kAbsTok, p.rows - t0), qp = p.dp + p.rp;
    const T *q = static_cast<const T *>(p.q) + (static_cast<size_t>(t0) * p.heads + h) * qp;
    const size_t qrow = static_cast<size_t>(p.heads) * qp;
    for (int e = tid; e < kAbsTok * p.dim; e += 256) {
        const int t = e / p.dim, d = e - t * p.dim;
        s_q[e] = t < toks ? dense::get(q + t * qrow + d) : 0.0f;
    }
    __syncthreads();
    const int cg = tid & 15, share = tid >> 4, col = c0 + cg * 8;
    float acc[kAbsTok][8] = {};
    if (col < p.uk_pitch) {
        const uint16_t *w = p.uk + static_cast<size_t>(h) * p.dim * p.uk_pitch + col;
#pragma unroll 4
        for (int d = share; d < p.dim; d += 16) {
            const uint4 v = *reinterpret_cast<const uint4 *>(w + static_cast<size_t>(d) * p.uk_pitch);
            const uint32_t wv[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
            for (int t = 0; t < kAbsTok; ++t) {
                const float x = s_q[t * p.dim + d];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    acc[t][2 * e] = fmaf(__uint_as_float(wv[e] << 16), x, acc[t][2 * e]);
                    acc[t][2 * e + 1] = fmaf(__uint_as_float(wv[e] & 0xffff0000u), x, acc[t][2 * e + 1]);
                }
            }
        }
    }
    const int warp = tid >> 5, lane = tid & 31;
#pragma unroll
    for (int t = 0; t < kAbsTok; ++t)
#pragma unroll
        for (int e = 0; e < 8; ++e) {
            const float v = acc[t][e] + __shfl_xor_sync(0xffffffffu, acc[t][e], 16);
            if (lane < 16) s_part[warp][t][cg * 8 + e] = v;
        }
    __syncthreads();
    T *ql = static_cast<T *>(p.ql) + (static_cast<size_t>(t0) * p.heads + h) * p.pitch;
    const size_t lrow = static_cast<size_t>(p.heads) * p.pitch;
    for (int e = tid; e < toks * kAbsCols; e += 256) {
        const int t = e / kAbsCols, c = e - t * kAbsCols;
        if (c0 + c >= p.kvp) continue;
        float v = 0.0f;
#pragma unroll
        for (int w = 0; w < 8; ++w) v += s_part[w][t][c];
        dense::put(ql + t * lrow + c0 + c, c0 + c < p.kv_rank ? v : 0.0f);
    }
    if (blockIdx.y == 0) {
        const int half = p.rot_dim / 2, pairs = p.rp / 2;
        for (int e = tid; e < toks * pairs; e += 256) {
            const int t = e / pairs, i = e - t * pairs;
            float a = 0.0f, b = 0.0f;
            if (i < half) {
                const float2 cs = turn(p.rot, i, p.rows_of_seq >= 0 ? p.pos[0] + t0 + t : p.pos[t0 + t]);
                const float u = dense::get(q + t * qrow + p.dp + 2 * i), v = dense::get(q + t * qrow + p.dp + 2 * i + 1);
                a = u * cs.x - v * cs.y;
                b = v * cs.x + u * cs.y;
            }
            dense::put(ql + t * lrow + p.kvp + 2 * i, a);
            dense::put(ql + t * lrow + p.kvp + 2 * i + 1, b);
        }
    }
}

// bf16: up to 16 rows of one head x 64 latent dimensions a block, on mma.sync: rows of queries are the M side, latent
// dimensions the N side (W_uk,h lies [dim][latent], which is the transposing load's form). Four warps, 16 dimensions each.
constexpr int kAbRows = 16, kAbCols = 64, kAbWarps = 4;
__global__ void __launch_bounds__(kAbWarps * 32) latent_absorb_mma_kernel(const QueryParams p) {
    extern __shared__ __align__(16) uint8_t ab_smem[];  // queries [16][dp * 2 + 16 bytes], weights [dp][64 * 2 + 16 bytes]
    const int h = blockIdx.x, c0 = blockIdx.y * kAbCols, t0 = blockIdx.z * kAbRows, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int toks = min(kAbRows, p.rows - t0), qp = p.dp + p.rp, qrow = p.dp * 2 + 16;
    constexpr int kWRow = kAbCols * 2 + 16;
    uint8_t *s_w = ab_smem + kAbRows * qrow;
    ptx::pdl_trigger();
    // the weights are constants: on their way while the kernel in front finishes
    for (int i = tid; i < p.dp * 8; i += kAbWarps * 32) {
        const int d = i >> 3, u = i & 7;
        uint8_t *dst = s_w + d * kWRow + u * 16;
        if (d < p.dim && c0 + u * 8 < p.uk_pitch) ptx::cp_async_16(ptx::smem_u32(dst), p.uk + (static_cast<size_t>(h) * p.dim + d) * p.uk_pitch + c0 + u * 8);
        else *reinterpret_cast<uint4 *>(dst) = make_uint4(0u, 0u, 0u, 0u);
    }
    ptx::cp_async_commit();
    ptx::pdl_wait();
    const uint16_t *q = static_cast<const uint16_t *>(p.q) + (static_cast<size_t>(t0) * p.heads + h) * qp;
    const size_t next = static_cast<size_t>(p.heads) * qp;
    for (int i = tid; i < kAbRows * (p.dp / 8); i += kAbWarps * 32) {
        const int r = i / (p.dp / 8), u = i - r * (p.dp / 8);
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (r < toks) v = *reinterpret_cast<const uint4 *>(q + r * next + u * 8);
        *reinterpret_cast<uint4 *>(ab_smem + r * qrow + u * 16) = v;
    }
    uint16_t *ql = static_cast<uint16_t *>(p.ql) + (static_cast<size_t>(t0) * p.heads + h) * p.pitch;
    const size_t lnext = static_cast<size_t>(p.heads) * p.pitch;
    if (blockIdx.y == 0) {
        const int half = p.rot_dim / 2, pairs = p.rp / 2;
        for (int e = tid; e < toks * pairs; e += kAbWarps * 32) {
            const int r = e / pairs, i = e - r * pairs;
            float a = 0.0f, b = 0.0f;
            if (i < half) {
                const float2 cs = turn(p.rot, i, p.rows_of_seq >= 0 ? p.pos[0] + t0 + r : p.pos[t0 + r]);
                const float u = dense::bf16_f32(q[r * next + p.dp + 2 * i]), v = dense::bf16_f32(q[r * next + p.dp + 2 * i + 1]);
                a = u * cs.x - v * cs.y;
                b = v * cs.x + u * cs.y;
            }
            *reinterpret_cast<uint32_t *>(ql + r * lnext + p.kvp + 2 * i) = dense::bf16_pair(a, b);
        }
    }
    ptx::cp_async_wait<0>();
    __syncthreads();
    const uint32_t q_lane = ptx::smem_u32(ab_smem) + ((lane & 7) + 8 * ((lane >> 3) & 1)) * qrow + (lane >> 4) * 16;
    const uint32_t w_lane = ptx::smem_u32(s_w) + ((lane & 7) + 8 * ((lane >> 3) & 1)) * kWRow + warp * 32 + (lane >> 4) * 16;
    float acc[2][4] = {};
    // what lies between dim and dp in the queries is a number or another layer's, and meets zeros
#pragma unroll 4
    for (int k = 0; k < p.dp; k += 16) {
        uint32_t a[4], b[4];
        ptx::ldmatrix_x4(a, q_lane + k * 2);
        ptx::ldmatrix_x4_trans(b, w_lane + k * kWRow);
        ptx::mma_bf16(acc[0], a, b[0], b[1]);
        ptx::mma_bf16(acc[1], a, b[2], b[3]);
    }
    const int g = lane >> 2, t = lane & 3;
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int tk = g + 8 * r, c = c0 + warp * 16 + n * 8 + 2 * t;  // columns past kv_rank have zero weights
            if (tk < toks && c < p.kvp) *reinterpret_cast<uint32_t *>(ql + tk * lnext + c) = dense::bf16_pair(acc[n][2 * r], acc[n][2 * r + 1]);
        }
}

// ---- attention over the latents, bf16 ---------------------------------------------------------------
using namespace tc;

constexpr int kLKeys = 64;          // positions at a time
constexpr int kLPiece = kLKeys * 128;  // bytes of 64 dimensions of them (SWIZZLE_128B)
constexpr int kLMaxPieces = 10, kLMaxLatent = 512;
constexpr int kLGroup = 8;          // heads of four warps; warp w: TMEM lane quadrant w % 4, heads of group w / 4
constexpr __host__ __device__ int latent_warps(int nh) { return 4 * nh / kLGroup; }  // and two more that issue copies and MMAs
constexpr float kLRescaleStep = 8.0f;  // in units of log 2
constexpr float kLog2e = 1.4426950408889634f;

struct LatentLayout {               // bytes from a 1024-byte boundary on
    int buf, q, p, misc, total;
    __host__ __device__ LatentLayout(int pieces, int nh) {
        buf = pieces * kLPiece;                // two of them
        q = 2 * buf;                           // the heads' queries, a piece [nh rows][128 bytes]
        p = q + pieces * nh * 128;             // probabilities, two buffers of [2 nh rows][64 positions]: high terms, then low
        misc = p + 2 * 2 * nh * 128;           // barriers, tensor memory address, abort flag, then maxima, reference maxima, factors
        total = misc + 256 + 3 * latent_warps(nh) * 32 * 4;
    }
};
struct LatentParams {
    CUtensorMap k;                  // bytes [sequences * cap][pitch * 2], box [64][128]
    CUtensorMap q;                  // bytes [rows * heads][pitch * 2], box [nh][128]
    const int *pos;
    int rows_of_seq, heads, width, kvp, cap, splits;
    float scale;                    // times log2(e)
    float *part;                    // [row][head][split][kvp + 4]
    int *err_word;
};

__device__ __forceinline__ void tmem_load(uint32_t at, uint32_t (&r)[8]) {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x8.b32 {%0,%1,%2,%3,%4,%5,%6,%7}, [%8];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7])
                 : "r"(at)
                 : "memory");
}
__device__ __forceinline__ void tmem_store(uint32_t at, const uint32_t (&r)[8]) {
    asm volatile("tcgen05.st.sync.aligned.32x32b.x8.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8};" ::"r"(at), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]),
                 "r"(r[6]), "r"(r[7])
                 : "memory");
}
// shared -> global, whole 16-byte units; the wait is until this thread's copies have been read from shared memory (they are
// complete when the grid is)
__device__ __forceinline__ void bulk_store(void *dst, uint32_t src, uint32_t bytes) {
    asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;\ncp.async.bulk.commit_group;" ::"l"(dst), "r"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void bulk_store_wait() { asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory"); }
// MN-major SWIZZLE_128B operand: 64 dimensions contiguous, groups of 8 positions 1024 bytes apart, pieces of 64 dimensions
// kLPiece apart
__device__ __forceinline__ uint64_t smem_desc_mn(uint32_t addr) {
    return static_cast<uint64_t>((addr & 0x3FFFFu) >> 4) | static_cast<uint64_t>(kLPiece >> 4) << 16 | static_cast<uint64_t>(1024 >> 4) << 32 | static_cast<uint64_t>(1) << 46 |
           static_cast<uint64_t>(2) << 61;
}
// MMAs and commits of a whole warp: every lane comes here with the same operands and one of them, always the same, issues.
// (Operands that are uniform over a converged warp sit in uniform registers, where the instruction wants them; under a
// branch of one lane each would have to be moved there first, which takes longer than these small MMAs do.)
__device__ __forceinline__ void umma(uint32_t d_tmem, uint64_t adesc, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n"
        ".reg .pred p, e;\n"
        "setp.ne.b32 p, %4, 0;\n"
        "elect.sync _|e, 0xffffffff;\n"
        "@e tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n"
        "}\n" ::"r"(d_tmem), "l"(adesc), "l"(bdesc), "r"(idesc), "r"(accumulate)
        : "memory");
}
// Four steps of it: the operands AS and BS (16-byte units) further each time.
template <int AS, int BS>
__device__ __forceinline__ void umma4(uint32_t d_tmem, uint64_t adesc, uint64_t bdesc, uint32_t idesc, uint32_t accumulate_first) {
    asm volatile(
        "{\n"
        ".reg .pred p, q, e;\n"
        ".reg .b64 a1, a2, a3, b1, b2, b3;\n"
        "setp.ne.b32 p, %4, 0;\n"
        "setp.eq.b32 q, 0, 0;\n"
        "add.u64 a1, %1, %5;\n"
        "add.u64 a2, %1, %6;\n"
        "add.u64 a3, %1, %7;\n"
        "add.u64 b1, %2, %8;\n"
        "add.u64 b2, %2, %9;\n"
        "add.u64 b3, %2, %10;\n"
        "elect.sync _|e, 0xffffffff;\n"
        "@e tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n"
        "@e tcgen05.mma.cta_group::1.kind::f16 [%0], a1, b1, %3, q;\n"
        "@e tcgen05.mma.cta_group::1.kind::f16 [%0], a2, b2, %3, q;\n"
        "@e tcgen05.mma.cta_group::1.kind::f16 [%0], a3, b3, %3, q;\n"
        "}\n" ::"r"(d_tmem), "l"(adesc), "l"(bdesc), "r"(idesc), "r"(accumulate_first), "n"(AS), "n"(2 * AS), "n"(3 * AS), "n"(BS), "n"(2 * BS), "n"(3 * BS)
        : "memory");
}
__device__ __forceinline__ void commit(uint32_t bar) {
    asm volatile(
        "{\n"
        ".reg .pred e;\n"
        "elect.sync _|e, 0xffffffff;\n"
        "@e tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];\n"
        "}\n" ::"r"(bar)
        : "memory");
}
__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// Over the 32 lanes, of N values each: lane l gets the maximum (or sum) of value l % N.
template <int N, bool MAX>
__device__ __forceinline__ float over_lanes(float (&v)[N], int lane) {
    auto both = [](float a, float b) { return MAX ? fmaxf(a, b) : a + b; };
#pragma unroll
    for (int w = N / 2; w >= 1; w >>= 1) {
        const bool up = (lane & w) != 0;
#pragma unroll
        for (int i = 0; i < w; ++i) v[i] = both(up ? v[i + w] : v[i], __shfl_xor_sync(0xffffffffu, up ? v[i] : v[i + w], w));
    }
    float t = v[0];
#pragma unroll
    for (int w = N; w < 32; w <<= 1) t = both(t, __shfl_xor_sync(0xffffffffu, t, w));
    return t;
}

template <int NH>  // heads a block takes, 16 or 32
__global__ void __launch_bounds__((latent_warps(NH) + 2) * 32, 1) latent_attn_kernel(const __grid_constant__ LatentParams p) {
    extern __shared__ uint8_t la_raw[];
    const uint32_t raw = ptx::smem_u32(la_raw), base = (raw + 1023u) & ~1023u;
    uint8_t *sm = la_raw + (base - raw);
    constexpr int HH = kLGroup, kLWarps = latent_warps(NH), kLTmaWarp = kLWarps, kLMmaWarp = kLWarps + 1;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int pieces = (p.width + 63) >> 6, blocks = (p.kvp + 127) >> 7;  // output blocks of 128 latent dimensions
    const LatentLayout L(pieces, NH);
    // Every barrier is a pair, by chunk parity: a wait for one chunk cannot be answered by the chunk two before it. Rows come
    // and go in parts of two pieces (128 dimensions): scores start on the first part while the others are on their way, and
    // a part is filled again as soon as its output block has been taken.
    const int parts = (pieces + 1) >> 1;
    constexpr int kParts = kLMaxPieces / 2, kFull = 0, kEmpty = 2 * kParts, kS = 4 * kParts, kP = kS + 2, kO = kS + 4;
    auto bar = [&](int kind, int j) { return base + L.misc + (kind + (j & 1)) * 8; };
    volatile uint32_t *s_tmem = reinterpret_cast<volatile uint32_t *>(sm + L.misc + 240);
    volatile int *s_abort = reinterpret_cast<volatile int *>(sm + L.misc + 244);
    float *s_max = reinterpret_cast<float *>(sm + L.misc + 256), *s_m = s_max + kLWarps * 32, *s_f = s_m + kLWarps * 32;
    if (tid == 0) {
        for (int i = 0; i < 2; ++i) {
            for (int k = 0; k < kParts; ++k) {
                ptx::mbar_init(bar(kFull + 2 * k, i), 1);
                ptx::mbar_init(bar(kEmpty + 2 * k, i), 1);
            }
            ptx::mbar_init(bar(kS, i), 1);
            ptx::mbar_init(bar(kP, i), kLWarps);
            ptx::mbar_init(bar(kO, i), 1);
        }
        *s_abort = 0;
        ptx::fence_barrier_init();
    }
    if (warp == kLMmaWarp) {
        tmem_alloc(base + L.misc + 240, 512);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    ptx::pdl_trigger();
    ptx::pdl_wait();
    const uint32_t t_s = *s_tmem, t_o = t_s + 2 * NH;        // two buffers of scores (NH columns), then per output block 2 NH: high and low terms' sums
    const int sp = blockIdx.x, h0 = blockIdx.y * NH, row = blockIdx.z, nh = min(NH, p.heads - h0);
    const int seq = p.rows_of_seq >= 0 ? p.rows_of_seq : row, pos = p.rows_of_seq >= 0 ? p.pos[0] + row : p.pos[row];
    const bool pos_ok = pos >= 0 && pos < p.cap;
    if (!pos_ok && tid == 0) atomicExch(p.err_word, 7);
    const int total = pos_ok ? pos + 1 : 0, per = ((total + p.splits - 1) / p.splits + kLKeys - 1) / kLKeys * kLKeys;
    const int u0 = min(total, sp * per), u1 = min(total, u0 + per), chunks = (u1 - u0 + kLKeys - 1) / kLKeys;
    const int prow = p.kvp + 4;
    bool ok = true;
    if (warp == kLTmaWarp) {
        if (lane == 0)
            for (int j = 0; j < chunks && ok; ++j)
                for (int k = 0; k < parts; ++k) {
                    if (j >= 2 && !wait_bar(bar(kEmpty + 2 * k, j), ((j >> 1) - 1) & 1, s_abort)) {
                        ok = false;
                        break;
                    }
                    const int p0 = 2 * k, p1 = min(pieces, p0 + 2);
                    ptx::mbar_arrive_expect_tx(bar(kFull + 2 * k, j), static_cast<uint32_t>((p1 - p0) * (kLPiece + (j ? 0 : NH * 128))));
                    for (int i = p0; i < p1; ++i) {
                        if (!j) ptx::tma_load_2d(base + L.q + i * NH * 128, &p.q, bar(kFull + 2 * k, 0), i * 128, row * p.heads + h0);
                        ptx::tma_load_2d(base + (j & 1) * L.buf + i * kLPiece, &p.k, bar(kFull + 2 * k, j), i * 128, seq * p.cap + u0 + j * kLKeys);
                    }
                }
    } else if (warp == kLMmaWarp) {
        if (chunks) {
            // D f32, A and B bf16, M = 128. Scores: the lower 64 rows of A are the positions, the upper 64 whatever lies behind them
            // (their lanes are not read). Output: A is MN-major (bit 15).
            constexpr uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((128u >> 4) << 24);
            constexpr uint32_t idesc_s = idesc | (static_cast<uint32_t>(NH >> 3) << 17), idesc_o = idesc | (1u << 15) | (static_cast<uint32_t>(2 * NH >> 3) << 17);
            const uint64_t k_desc = smem_desc_sw128(base), q_desc = smem_desc_sw128(base + L.q), v_desc = smem_desc_mn(base), p_desc = smem_desc_sw128(base + L.p);
            const int ksteps = p.width >> 4;
            const uint32_t u_s = __shfl_sync(0xffffffffu, t_s, 0), u_o = u_s + 2 * NH;
            auto scores = [&](int j, int k) {                // of part k's dimensions
                const uint64_t kd = k_desc + static_cast<uint64_t>((j & 1) * (L.buf >> 4));
                const int end = min(ksteps, 8 * k + 8);
                uint64_t a = kd + static_cast<uint64_t>(2 * k * (kLPiece >> 4)), b = q_desc + static_cast<uint64_t>(2 * k * (NH * 128 >> 4));
                int st = 8 * k;
#pragma unroll
                for (int i = 0; i < 2; ++i)                  // pieces of 64 dimensions
                    if (st + 4 <= end) {
                        umma4<2, 2>(u_s + (j & 1) * NH, a, b, idesc_s, (k | i) ? 1u : 0u);
                        a += kLPiece >> 4;
                        b += NH * 128 >> 4;
                        st += 4;
                    }
                for (; st < end; ++st)
                    umma(u_s + (j & 1) * NH, kd + static_cast<uint64_t>((st >> 2) * (kLPiece >> 4) + (st & 3) * 2),
                         q_desc + static_cast<uint64_t>((st >> 2) * (NH * 128 >> 4) + (st & 3) * 2), idesc_s, st ? 1u : 0u);
                if (k == parts - 1) commit(bar(kS, j));
            };
            auto values = [&](int j) {
                const uint64_t vd = v_desc + static_cast<uint64_t>((j & 1) * (L.buf >> 4)), pd = p_desc + static_cast<uint64_t>((j & 1) * (2 * NH * 128 >> 4));
                for (int k = 0; k < parts; ++k) {
                    if (k < blocks) umma4<(2048 >> 4), 2>(u_o + k * 2 * NH, vd + static_cast<uint64_t>(k * (2 * kLPiece >> 4)), pd, idesc_o, j ? 1u : 0u);  // 16 positions a step
                    commit(bar(kEmpty + 2 * k, j));
                }
                commit(bar(kO, j));
            };
            // Values of chunk nv as soon as its probabilities are there, else scores of chunk ns's next part as soon as that
            // is, never more than two chunks apart. So scores of j + 1 go after values of j - 1: the probabilities of j - 1
            // mean that its scores have been read (the buffer is j + 1's), and scores of j + 1 mean that the probabilities
            // of j - 1 have been (the same for theirs).
            int ns = 0, nk = 0, nv = 0;
            uint32_t idle = 0;
            while (nv < chunks) {
                if (nv < ns && __all_sync(0xffffffffu, ptx::mbar_test_wait(bar(kP, nv), (nv >> 1) & 1))) {
                    tc_fence_after();
                    values(nv++);
                    idle = 0;
                } else if (ns < chunks && ns <= nv + 1 && __all_sync(0xffffffffu, ptx::mbar_test_wait(bar(kFull + 2 * nk, ns), (ns >> 1) & 1))) {
                    scores(ns, nk);
                    if (++nk == parts) {
                        nk = 0;
                        ++ns;
                    }
                    idle = 0;
                } else if (__any_sync(0xffffffffu, *s_abort || ++idle > kTcWaitLimit)) {
                    *s_abort = 1;
                    ok = false;
                    break;
                }
            }
        }
    } else {
        auto wait_all = [&](uint32_t b, uint32_t parity) { return __all_sync(0xffffffffu, wait_bar(b, parity, s_abort)) != 0; };
        const int quad = warp & 3, group = warp >> 2;        // positions are in quadrants 0 and 1; all four hold latent dimensions
        const uint32_t lanes = static_cast<uint32_t>(quad * 32) << 16;
        auto meet = [&]() { asm volatile("bar.sync %0, 128;" ::"r"(1 + group) : "memory"); };  // the four warps of a group
        float *w_m = s_m + warp * 32, *w_f = s_f + warp * 32, *g_max = s_max + group * 4 * 32;
        float m = -1e30f, l = 0.0f;                          // of head lane % HH: the maximum probabilities are scaled with, this warp's share of the sum
        // Every warp comes to the meeting of a chunk and to the one after the loop whatever a wait returned: a warp whose
        // wait gave up skips the work, never the meetings.
        for (int j = 0; j < chunks; ++j) {
            const int key = u0 + j * kLKeys + quad * 32 + lane;
            float s[HH], v[HH];
            if (quad < 2) {
                if (ok && !wait_all(bar(kS, j), (j >> 1) & 1)) ok = false;
                if (ok) {
                    tc_fence_after();
                    uint32_t r[HH];
                    tmem_load(t_s + (j & 1) * NH + group * HH + lanes, r);
                    tmem_ld_wait();
#pragma unroll
                    for (int i = 0; i < HH; ++i) s[i] = v[i] = key < u1 ? __uint_as_float(r[i]) * p.scale : -INFINITY;
                    g_max[((j & 1) * 2 + quad) * 32 + lane] = over_lanes<HH, true>(v, lane);
                }
            }
            meet();  // the maxima's place of this parity is written again two chunks later, after the next meeting
            if (!ok) continue;
            const float mx = fmaxf(g_max[(j & 1) * 2 * 32 + lane], g_max[((j & 1) * 2 + 1) * 32 + lane]);  // finite: a chunk has a position
            const float nm = mx > m + kLRescaleStep ? mx : m, corr = ex2(m - nm);
            const bool moved = __any_sync(0xffffffffu, nm != m) && j > 0;  // the same in the four warps
            m = nm;
            w_m[lane] = nm;
            w_f[lane] = corr;
            __syncwarp();
            if (moved) {                                     // nothing adds to the output before all warps say that their probabilities are ready
                if (!wait_all(bar(kO, j - 1), ((j - 1) >> 1) & 1)) {
                    ok = false;
                    continue;
                }
                tc_fence_after();
                for (int c = 0; c < 2 * blocks; ++c) {       // high and low terms of every block
                    uint32_t r[HH];
                    tmem_load(t_o + c * NH + group * HH + lanes, r);
                    tmem_ld_wait();
#pragma unroll
                    for (int i = 0; i < HH; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * w_f[i]);
                    tmem_store(t_o + c * NH + group * HH + lanes, r);
                }
                tmem_st_wait();
            }
            if (quad < 2) {
                // position k of head i: row i, 16-byte unit k / 8 XOR-ed with i % 8
                const int k = quad * 32 + lane;
                uint8_t *pp = sm + L.p + (j & 1) * 2 * NH * 128 + group * HH * 128 + (k & 6) * 2;
                const bool odd = (lane & 1) != 0;
                uint32_t both[HH];                           // high term, low term
#pragma unroll
                for (int i = 0; i < HH; ++i) {
                    const float e = ex2(s[i] - w_m[i]);
                    v[i] = e;
                    const float hi = __uint_as_float(dense::bf16_pair(e, 0.0f) << 16);
                    both[i] = dense::bf16_pair(hi, e - hi);
                }
                // neighbouring lanes hold neighbouring positions: one writes both of head i, the other both of head i + 1
#pragma unroll
                for (int i = 0; i < HH; i += 2) {
                    const uint32_t got = __shfl_xor_sync(0xffffffffu, odd ? both[i] : both[i + 1], 1), own = odd ? both[i + 1] : both[i];
                    const uint32_t first = odd ? got : own, second = odd ? own : got;
                    const int head = i + (odd ? 1 : 0);
                    uint8_t *at = pp + head * 128 + (((k >> 3) ^ (head & 7)) << 4);
                    *reinterpret_cast<uint32_t *>(at) = __byte_perm(first, second, 0x5410);
                    *reinterpret_cast<uint32_t *>(at + NH * 128) = __byte_perm(first, second, 0x7632);
                }
                l = l * corr + over_lanes<HH, false>(v, lane);
                if (key >= total && group == 0) {             // nothing has been written there: its weight is zero, but the bits must be numbers
                    for (int i = 0; i < pieces; ++i)
#pragma unroll
                        for (int u = 0; u < 8; ++u) *reinterpret_cast<uint4 *>(sm + (j & 1) * L.buf + i * kLPiece + k * 128 + u * 16) = make_uint4(0u, 0u, 0u, 0u);
                }
                ptx::fence_proxy_async();
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) ptx::mbar_arrive(bar(kP, j));
        }
        if (ok && chunks && !wait_all(bar(kO, chunks - 1), ((chunks - 1) >> 1) & 1)) ok = false;
        tc_fence_after();
        // this slice's sums and, unscaled, the weighted latents (an empty slice: no weight, zeros)
        w_f[lane] = l;
        float *out = reinterpret_cast<float *>(sm) + group * HH * p.kvp;  // every copy and MMA has finished: the rows' buffers are free
        for (int db = 0; db < blocks; ++db) {
            uint32_t r[HH], lo[HH];
#pragma unroll
            for (int i = 0; i < HH; ++i) r[i] = lo[i] = 0;
            if (ok && chunks) {
                tmem_load(t_o + db * 2 * NH + group * HH + lanes, r);
                tmem_load(t_o + db * 2 * NH + NH + group * HH + lanes, lo);
                tmem_ld_wait();
            }
            const int d = db * 128 + quad * 32 + lane;
            if (d < p.kvp)
#pragma unroll
                for (int i = 0; i < HH; ++i) out[i * p.kvp + d] = __uint_as_float(r[i]) + __uint_as_float(lo[i]);
        }
        ptx::fence_proxy_async();
        meet();
        if (quad == 0 && lane < HH && group * HH + lane < nh) {
            float *dst = p.part + ((static_cast<size_t>(row) * p.heads + h0 + group * HH + lane) * p.splits + sp) * prow;
            bulk_store(dst, ptx::smem_u32(out + lane * p.kvp), static_cast<uint32_t>(p.kvp) * 4);
            dst[p.kvp] = chunks ? m / kLog2e : -INFINITY;
            dst[p.kvp + 1] = w_f[lane] + w_f[32 + lane];  // this warp's and the next one's
            bulk_store_wait();
        }
        tc_fence_before();
    }
    if (!ok && lane == 0) atomicExch(p.err_word, 5);
    __syncthreads();
    if (warp == kLMmaWarp) {
        tc_fence_after();
        tmem_dealloc(t_s, 512);
    }
}

// ---- out: merge, W_uv, gate -----------------------------------------------------------------------------
struct OutParams {
    const float *part;              // slices, or (32-bit) the weighted latents themselves, [row][heads][kv_rank]
    int rows, heads, splits, vdim, kv_rank, kvp;
    const uint16_t *uv;
    int uv_pitch, vrows;            // vrows: value dimensions a block takes (a multiple of 16)
    const float *gate;
    long ldg, ldo;
    void *out;
};
constexpr int kMergeTok = 8;        // the MMA's N side
__global__ void __launch_bounds__(256) latent_merge_kernel(const OutParams p) {
    __shared__ __align__(16) float s_sum[8][kLMaxLatent];    // [warp][latent]
    __shared__ __align__(16) uint16_t s_x[kMergeTok][kLMaxLatent + 32];  // eight rows start in different bank groups
    ptx::pdl_trigger();
    const int h = blockIdx.x, e0 = blockIdx.y * p.vrows, t0 = blockIdx.z * kMergeTok, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int toks = min(kMergeTok, p.rows - t0), prow = p.kvp + 4;
    // the weights are constants: the warp's first 16 rows are on their way while the kernel in front finishes
    const int g = lane >> 2, t = lane & 3, e_end = min(p.vdim, e0 + p.vrows);
    constexpr int kAhead = 8;
    uint4 wl[kAhead], wh[kAhead];
    auto weights = [&](int r0, int c0) {                     // 32 columns each: 16 bytes a lane are two MMAs' operands
        const uint16_t *lo = p.uv + static_cast<size_t>(h * p.vdim + min(r0 + g, p.vdim - 1)) * p.uv_pitch + t * 8;
        const uint16_t *hi = p.uv + static_cast<size_t>(h * p.vdim + min(r0 + g + 8, p.vdim - 1)) * p.uv_pitch + t * 8;
#pragma unroll
        for (int i = 0; i < kAhead; ++i)
            if (c0 + 32 * i < p.uv_pitch) {
                wl[i] = *reinterpret_cast<const uint4 *>(lo + c0 + 32 * i);
                wh[i] = *reinterpret_cast<const uint4 *>(hi + c0 + 32 * i);
            }
    };
    if (e0 + warp * 16 < e_end) weights(e0 + warp * 16, 0);
    ptx::pdl_wait();
    // a warp or several for each row, every so many slices; what lies between kv_rank and kvp is zero
    int share = 8;
    while (share * toks > 8) share >>= 1;
    const int tok = warp / share, sub = warp - tok * share;
    if (tok < toks) {
        const float *part = p.part + (static_cast<size_t>(t0 + tok) * p.heads + h) * p.splits * prow;
        const int sa = lane, sb = lane + 32;                 // at most 64 slices
        const float ma = sa < p.splits ? part[static_cast<size_t>(sa) * prow + p.kvp] : -INFINITY, mb = sb < p.splits ? part[static_cast<size_t>(sb) * prow + p.kvp] : -INFINITY;
        const float la = sa < p.splits ? part[static_cast<size_t>(sa) * prow + p.kvp + 1] : 0.0f, lb = sb < p.splits ? part[static_cast<size_t>(sb) * prow + p.kvp + 1] : 0.0f;
        float4 a[kLMaxLatent / 128];
#pragma unroll
        for (int j = 0; j < kLMaxLatent / 128; ++j) a[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        float wa = 0.0f, wb = 0.0f;
        constexpr int kBatch = 5;                            // slices whose values are in flight together
        for (int s0 = sub; s0 < p.splits; s0 += kBatch * share) {
            float4 v[kBatch][kLMaxLatent / 128];
#pragma unroll
            for (int k = 0; k < kBatch; ++k)
#pragma unroll
                for (int j = 0; j < kLMaxLatent / 128; ++j) {
                    const int s = s0 + k * share;
                    v[k][j] = make_float4(0.f, 0.f, 0.f, 0.f);
                    if (s < p.splits && lane * 4 + 128 * j < p.kvp) v[k][j] = *reinterpret_cast<const float4 *>(part + static_cast<size_t>(s) * prow + lane * 4 + 128 * j);
                }
            if (s0 == sub) {
                float mx = fmaxf(ma, mb);
#pragma unroll
                for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
                wa = ma == -INFINITY ? 0.0f : __expf(ma - mx);
                wb = mb == -INFINITY ? 0.0f : __expf(mb - mx);
                float sum = wa * la + wb * lb;
#pragma unroll
                for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
                wa /= sum;
                wb /= sum;
            }
#pragma unroll
            for (int k = 0; k < kBatch; ++k) {
                const int s = s0 + k * share;
                const float x = __shfl_sync(0xffffffffu, s < 32 ? wa : wb, s & 31), w = s < p.splits ? x : 0.0f;
#pragma unroll
                for (int j = 0; j < kLMaxLatent / 128; ++j) {
                    a[j].x = fmaf(w, v[k][j].x, a[j].x); a[j].y = fmaf(w, v[k][j].y, a[j].y); a[j].z = fmaf(w, v[k][j].z, a[j].z); a[j].w = fmaf(w, v[k][j].w, a[j].w);
                }
            }
        }
#pragma unroll
        for (int j = 0; j < kLMaxLatent / 128; ++j) {
            if (share == 1) dense::put4(&s_x[tok][lane * 4 + 128 * j], a[j]);
            else *reinterpret_cast<float4 *>(&s_sum[warp][lane * 4 + 128 * j]) = a[j];
        }
    }
    if (share > 1) __syncthreads();
    for (int i = tid; i < kMergeTok * p.uv_pitch; i += 256) {
        const int tk = i / p.uv_pitch, c = i - tk * p.uv_pitch;
        if (tk < toks && share == 1) continue;               // already there
        float v = 0.0f;
        if (tk < toks)
            for (int k = 0; k < share; ++k) v += s_sum[tk * share + k][c];
        s_x[tk][c] = dense::f32_bf16(v);
    }
    __syncthreads();
    for (int r0 = e0 + warp * 16; r0 < e_end; r0 += 128) {
        float acc[4] = {0.0f, 0.0f, 0.0f, 0.0f};
        for (int c0 = 0; c0 < p.uv_pitch; c0 += 32 * kAhead) {
            if (c0 || r0 != e0 + warp * 16) weights(r0, c0);
#pragma unroll
            for (int i = 0; i < kAhead; ++i)
                if (c0 + 32 * i < p.uv_pitch) {
                    const uint4 b = *reinterpret_cast<const uint4 *>(&s_x[g][c0 + 32 * i + t * 8]);
                    const uint32_t a0[4] = {wl[i].x, wh[i].x, wl[i].y, wh[i].y}, a1[4] = {wl[i].z, wh[i].z, wl[i].w, wh[i].w};
                    ptx::mma_bf16(acc, a0, b.x, b.y);        // both operands with the same order of columns
                    ptx::mma_bf16(acc, a1, b.z, b.w);
                }
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int tk = 2 * t + (i & 1), e = r0 + g + 8 * (i >> 1);
            if (tk < toks && e < e_end)
                static_cast<uint16_t *>(p.out)[static_cast<size_t>(t0 + tk) * p.ldo + static_cast<size_t>(h) * p.vdim + e] =
                    dense::f32_bf16(acc[i] * dense::sigmoid(p.gate[static_cast<size_t>(t0 + tk) * p.ldg + h]));
        }
    }
}

constexpr int kOutTok = 4, kOutRows = 32;
__global__ void __launch_bounds__(256) latent_out_kernel(const OutParams p) {
    ptx::pdl_trigger();
    ptx::pdl_wait();
    extern __shared__ float s_dyn[];                         // [kOutTok][uv_pitch]
    const int h = blockIdx.x, e0 = blockIdx.y * kOutRows, t0 = blockIdx.z * kOutTok, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int toks = min(kOutTok, p.rows - t0);
    for (int i = tid; i < kOutTok * p.uv_pitch; i += 256) {
        const int t = i / p.uv_pitch, c = i - t * p.uv_pitch;
        s_dyn[i] = t < toks && c < p.kv_rank ? p.part[(static_cast<size_t>(t0 + t) * p.heads + h) * p.kv_rank + c] : 0.0f;
    }
    __syncthreads();
    for (int r = warp; r < kOutRows; r += 8) {
        const int e = e0 + r;
        if (e >= p.vdim) break;
        const uint16_t *w = p.uv + static_cast<size_t>(h * p.vdim + e) * p.uv_pitch;
        float acc[kOutTok] = {};
        for (int i = lane; i < p.uv_pitch; i += 32) {
            const float wv = dense::bf16_f32(w[i]);
#pragma unroll
            for (int t = 0; t < kOutTok; ++t) acc[t] = fmaf(wv, s_dyn[t * p.uv_pitch + i], acc[t]);
        }
#pragma unroll
        for (int t = 0; t < kOutTok; ++t) {
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) acc[t] += __shfl_xor_sync(0xffffffffu, acc[t], o);
            if (lane == 0 && t < toks)
                static_cast<float *>(p.out)[static_cast<size_t>(t0 + t) * p.ldo + static_cast<size_t>(h) * p.vdim + e] =
                    acc[t] * dense::sigmoid(p.gate[static_cast<size_t>(t0 + t) * p.ldg + h]);
        }
    }
}

constexpr size_t kMaxSplits = 64;
constexpr int kLatentSmem = 227 * 1024;
static_assert(kMaxSplits <= 64, "a lane of the merge holds two slices' weights");

// The scores' operand is read 128 rows at a time (half of them belong to what lies behind a piece), the output's in blocks of
// two pieces: all of it has to be the block's own shared memory.
int latent_smem(const LatentShape &s, int nh) {
    const int pieces = static_cast<int>((s.kvp() + s.rp() + 63) / 64), own = LatentLayout(pieces, nh).total;
    const int scores = (2 * pieces + 1) * kLPiece, values = pieces * kLPiece + static_cast<int>((s.kvp() + 127) / 128) * 2 * kLPiece;
    return std::max(own, std::max(scores, values)) + 1024;
}

int latent_init(Ctx *ctx) {
    const int most = static_cast<int>(ctx->smem_optin) < kLatentSmem ? static_cast<int>(ctx->smem_optin) : kLatentSmem;
    LBK_CUDA(cudaFuncSetAttribute(latent_absorb_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, most));
    LBK_CUDA(cudaFuncSetAttribute(latent_attn_kernel<16>, cudaFuncAttributeMaxDynamicSharedMemorySize, most));
    LBK_CUDA(cudaFuncSetAttribute(latent_attn_kernel<32>, cudaFuncAttributeMaxDynamicSharedMemorySize, most));
    return LBK_OK;
}
const InitHook kInitLatent(latent_init);

int check_shape(const LatentShape &s) {
    if (!s.heads || !s.dim || !s.rot_dim || s.rot_dim % 2 || !s.vdim || !s.kv_rank || !s.q_rank) return fail(LBK_ERR_SHAPE, "latent attention: a size is zero or the rotated part is odd");
    if (s.kvp() + s.rp() > 1024) return fail(LBK_ERR_UNSUPPORTED, "latent attention: latent and rotated part of at most 1024 values");
    if (s.dim > 1024 || s.vdim > 1024) return fail(LBK_ERR_UNSUPPORTED, "latent attention: head sizes of at most 1024");
    return LBK_OK;
}

QueryParams query_params(const LatentAttnCall &c) {
    QueryParams p{};
    p.q = c.q;
    p.ql = c.ql;
    p.rows = static_cast<int>(c.rows);
    p.rows_of_seq = c.rows_of_seq;
    p.heads = static_cast<int>(c.s.heads);
    p.dim = static_cast<int>(c.s.dim);
    p.dp = static_cast<int>(c.s.dp());
    p.rot_dim = static_cast<int>(c.s.rot_dim);
    p.rp = static_cast<int>(c.s.rp());
    p.kv_rank = static_cast<int>(c.s.kv_rank);
    p.kvp = static_cast<int>(c.s.kvp());
    p.pitch = static_cast<int>(c.s.pitch());
    p.pos = c.pos;
    p.rot = angles(c.rot);
    p.uk = c.uk.w;
    p.uk_pitch = static_cast<int>(c.uk.pitch);
    return p;
}

}  // namespace

void rotation_frequencies(size_t dims, double base, const YarnScaling &y, double *freq, float *factor) {
    for (size_t i = 0; i < dims / 2; ++i) freq[i] = std::pow(base, -2.0 * static_cast<double>(i) / static_cast<double>(dims));
    *factor = 1.0f;
    if (!y.on) return;
    const double n = static_cast<double>(dims), pi = 3.14159265358979323846;
    auto turns = [&](double t) { return n * std::log(y.original / (2.0 * pi * t)) / (2.0 * std::log(base)); };
    const double lo = std::max(std::floor(turns(y.fast)), 0.0), hi = std::min(std::ceil(turns(y.slow)), n - 1.0);
    for (size_t i = 0; i < dims / 2; ++i) {
        const double ramp = std::min(std::max((static_cast<double>(i) - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
        freq[i] = freq[i] / y.factor * ramp + freq[i] * (1.0 - ramp);
    }
    *factor = static_cast<float>(0.1 * std::log(y.factor) + 1.0);
}

int launch_latent_prep(Ctx *ctx, const LatentPrepCall &c, cudaStream_t st) {
    if (c.rows == 0) return LBK_OK;
    LBK_TRY(check_shape(c.s));
    if (!c.z || !c.cq || !c.q_norm || (c.cache && (!c.kv_norm || !c.pos || !c.rot.freq))) return fail(LBK_ERR_INVALID, "latent attention: null buffer");
    PrepParams p{};
    p.z = c.z;
    p.ldz = c.ldz;
    p.ldq = c.ldq;
    p.q_rank = static_cast<int>(c.s.q_rank);
    p.kv_rank = static_cast<int>(c.s.kv_rank);
    p.rot_dim = static_cast<int>(c.s.rot_dim);
    p.kvp = static_cast<int>(c.s.kvp());
    p.pitch = static_cast<int>(c.s.pitch());
    p.rows = static_cast<int>(c.rows);
    p.rows_of_seq = c.rows_of_seq;
    p.cap = static_cast<int>(c.cap);
    p.pos = c.pos;
    p.q_norm = c.q_norm;
    p.kv_norm = c.kv_norm;
    p.eps = c.eps;
    p.rot = angles(c.rot);
    p.cq = c.cq;
    p.cache = c.cache;
    p.err_word = ctx->err_word;
    LBK_CUDA(launch_chained(c.compute == LBK_COMPUTE_F32 ? latent_prep_kernel<float> : latent_prep_kernel<uint16_t>, dim3(static_cast<unsigned>(c.rows)), dim3(256), 0, st, p));
    LBK_CUDA(cudaGetLastError());
    ctx->launches++;
    return LBK_OK;
}

size_t latent_splits(size_t cap) {
    const size_t s = (cap + kLKeys - 1) / kLKeys;
    return s < 1 ? 1 : s > kMaxSplits ? kMaxSplits : s;
}
// slices of the weighted latents (rows x slices stays near the number of SMs), or (32-bit) the weighted latents
size_t latent_scratch(const Ctx *ctx, size_t rows, const LatentShape &s, size_t splits) {
    return s.heads * std::min(rows * splits, rows + static_cast<size_t>(ctx->sm_count)) * (s.kvp() + 4);
}

int launch_latent_absorbed(Ctx *ctx, const LatentAttnCall &c, cudaStream_t st) {
    if (c.rows == 0) return LBK_OK;
    LBK_TRY(check_shape(c.s));
    if (!c.q || !c.ql || !c.cache || !c.pos || !c.scratch || !c.uk.w || !c.uv.w || !c.gate || !c.out || !c.splits) return fail(LBK_ERR_INVALID, "latent attention: null buffer");
    if (c.rows > 65535) return fail(LBK_ERR_UNSUPPORTED, "at most 65535 rows per call");
    const bool f32 = c.compute == LBK_COMPUTE_F32;
    const QueryParams qp = query_params(c);
    if (f32) {
        const dim3 grid(static_cast<unsigned>(c.s.heads), static_cast<unsigned>((c.s.kvp() + kAbsCols - 1) / kAbsCols), static_cast<unsigned>((c.rows + kAbsTok - 1) / kAbsTok));
        LBK_CUDA(launch_chained(latent_absorb_kernel, grid, dim3(256), kAbsTok * c.s.dim * sizeof(float), st, qp));
    } else {
        const dim3 grid(static_cast<unsigned>(c.s.heads), static_cast<unsigned>((c.s.kvp() + kAbCols - 1) / kAbCols), static_cast<unsigned>((c.rows + kAbRows - 1) / kAbRows));
        LBK_CUDA(launch_chained(latent_absorb_mma_kernel, grid, dim3(kAbWarps * 32), kAbRows * (c.s.dp() * 2 + 16) + c.s.dp() * (kAbCols * 2 + 16), st, qp));
    }
    LBK_CUDA(cudaGetLastError());
    ctx->launches++;
    OutParams op{};
    op.part = c.scratch;
    op.rows = qp.rows;
    op.heads = qp.heads;
    op.vdim = static_cast<int>(c.s.vdim);
    op.kv_rank = qp.kv_rank;
    op.kvp = qp.kvp;
    op.uv = c.uv.w;
    op.uv_pitch = static_cast<int>(c.uv.pitch);
    op.gate = c.gate;
    op.ldg = c.ldg;
    op.ldo = c.ldo;
    op.out = c.out;
    if (f32) {
        // the general kernel: one key / value head whose values are the front of its keys
        AttnCall a;
        a.compute = c.compute;
        a.q = c.ql;
        a.kc = a.vc = c.cache;
        a.pos = c.pos;
        a.n = c.rows;
        a.rows_of_seq = c.rows_of_seq;
        a.heads = c.s.heads;
        a.kv_heads = 1;
        a.dim = c.s.kvp() + c.s.rp();
        a.vdim = c.s.kv_rank;
        a.dimp = a.vdimp = c.s.pitch();
        a.cap = c.cap;
        a.scale = c.scale;
        a.mask.alibi = false;
        a.out = c.scratch;
        a.ldo = static_cast<long>(c.s.heads * c.s.kv_rank);
        LBK_TRY(launch_attn_window(ctx, a, st));
    } else {
        const int nh = c.s.heads > 16 ? 32 : 16;
        if (!latent_absorb_supported(c.s)) return fail(LBK_ERR_UNSUPPORTED, "latent attention in bf16: latents of at most %d values, rotated parts of at most 128", kLMaxLatent);
        LatentParams p{};
        const size_t pitch = c.s.pitch() * 2, seqs = c.rows_of_seq >= 0 ? static_cast<size_t>(c.rows_of_seq) + 1 : c.rows;
        LBK_TRY(encode_bytes_map(&p.k, c.cache, pitch, seqs * c.cap, pitch, 128, kLKeys));
        LBK_TRY(encode_bytes_map(&p.q, c.ql, pitch, c.rows * c.s.heads, pitch, 128, nh));
        p.pos = c.pos;
        p.rows_of_seq = c.rows_of_seq;
        p.heads = qp.heads;
        p.width = static_cast<int>(c.s.kvp() + c.s.rp());
        p.kvp = qp.kvp;
        p.cap = static_cast<int>(c.cap);
        p.scale = c.scale * kLog2e;
        p.part = c.scratch;
        p.err_word = ctx->err_word;
        const size_t tiles = (c.s.heads + nh - 1) / nh;
        // about one block per SM: as many slices as that leaves
        const size_t want = static_cast<size_t>(ctx->sm_count) / (c.rows * tiles);
        p.splits = static_cast<int>(want < 1 ? 1 : want < c.splits ? want : c.splits);
        op.splits = p.splits;
        const dim3 grid(static_cast<unsigned>(p.splits), static_cast<unsigned>(tiles), static_cast<unsigned>(c.rows));
        LBK_CUDA(launch_chained(nh == 32 ? latent_attn_kernel<32> : latent_attn_kernel<16>, grid, dim3(static_cast<unsigned>(latent_warps(nh) + 2) * 32), static_cast<size_t>(latent_smem(c.s, nh)), st, p));
        LBK_CUDA(cudaGetLastError());
        ctx->launches++;
        // a block for eight rows of a head, or for fewer value dimensions of them when that leaves SMs idle
        const size_t ttiles = (c.rows + kMergeTok - 1) / kMergeTok, vtiles = (c.s.vdim + 15) / 16;
        size_t parts = static_cast<size_t>(ctx->sm_count) / (c.s.heads * ttiles);
        parts = parts < 1 ? 1 : parts > vtiles ? vtiles : parts;
        op.vrows = static_cast<int>((vtiles + parts - 1) / parts * 16);
        const dim3 mgrid(static_cast<unsigned>(c.s.heads), static_cast<unsigned>((c.s.vdim + op.vrows - 1) / op.vrows), static_cast<unsigned>(ttiles));
        LBK_CUDA(launch_chained(latent_merge_kernel, mgrid, dim3(256), 0, st, op));
        LBK_CUDA(cudaGetLastError());
        ctx->launches++;
        return LBK_OK;
    }
    const dim3 ogrid(static_cast<unsigned>(c.s.heads), static_cast<unsigned>((c.s.vdim + kOutRows - 1) / kOutRows), static_cast<unsigned>((c.rows + kOutTok - 1) / kOutTok));
    LBK_CUDA(launch_chained(latent_out_kernel, ogrid, dim3(256), kOutTok * c.uv.pitch * sizeof(float), st, op));
    LBK_CUDA(cudaGetLastError());
    ctx->launches++;
    return LBK_OK;
}

bool latent_absorb_supported(const LatentShape &s) {
    return s.kvp() <= kLMaxLatent && (s.kvp() + s.rp() + 63) / 64 <= kLMaxPieces && latent_smem(s, 32) <= kLatentSmem;
}
bool latent_expand_supported(const LatentShape &s) { return (s.dp() + 63) / 64 + (s.rp() + 63) / 64 <= 3 && s.vp() <= 128; }

int launch_latent_expanded(Ctx *ctx, const LatentAttnCall &c, cudaStream_t st) {
    if (c.rows == 0) return LBK_OK;
    LBK_TRY(check_shape(c.s));
    if (c.compute != LBK_COMPUTE_BF16 || c.rows_of_seq < 0 || !latent_expand_supported(c.s)) return fail(LBK_ERR_INVALID, "latent attention: these rows cannot take the expanding form");
    if (!c.q || !c.cache || !c.pos || !c.ek || !c.ev || !c.ukv.w || !c.gate || !c.zero || !c.out || c.ecap < c.length || c.length > c.cap) return fail(LBK_ERR_INVALID, "latent attention: null or short buffer");
    const uint16_t *rows = static_cast<const uint16_t *>(c.cache) + static_cast<size_t>(c.rows_of_seq) * c.cap * c.s.pitch();
    DenseCall d;
    d.compute = c.compute;
    d.x = rows;
    d.ldx = static_cast<long>(c.s.pitch());
    d.m = c.length;
    d.w = c.ukv;
    d.out_rows = c.ukv.rows;
    d.epi.kind = kEpiQkv;
    d.epi.k_rows = static_cast<int>(c.s.heads * c.s.dim);
    d.epi.dim = static_cast<int>(c.s.dim);
    d.epi.dimp = static_cast<int>(c.s.dp());
    d.epi.vdim = static_cast<int>(c.s.vdim);
    d.epi.vdimp = static_cast<int>(c.s.vp());
    d.epi.kv_heads = static_cast<int>(c.s.heads);
    d.epi.cap = static_cast<int>(c.ecap);
    d.epi.kc = c.ek;
    d.epi.vc = c.ev;
    d.epi.pos = c.zero;
    d.epi.rows_of_seq = 0;
    d.epi.err_word = ctx->err_word;
    LBK_TRY(launch_dense(ctx, d, st));
    const QueryParams qp = query_params(c);
    LBK_CUDA(launch_chained(latent_rotate_kernel<uint16_t>, dim3(static_cast<unsigned>(c.rows)), dim3(256), c.s.rot_dim / 2 * sizeof(float2), st, qp));
    LBK_CUDA(cudaGetLastError());
    ctx->launches++;
    AttnCall a;
    a.q = c.q;
    a.kc = c.ek;
    a.vc = c.ev;
    a.pos = c.pos;
    a.n = c.rows;
    a.rows_of_seq = 0;
    a.heads = a.kv_heads = c.s.heads;
    a.dim = c.s.dim;
    a.dimp = c.s.dp();
    a.vdim = c.s.vdim;
    a.vdimp = c.s.vp();
    a.cap = c.ecap;
    a.scale = c.scale;
    a.mask.alibi = false;
    a.k2 = rows + c.s.kvp();
    a.dim2p = c.s.rp();
    a.k2_pitch = c.s.pitch();
    a.k2_rows = c.length;
    a.gate = c.gate;
    a.ldg = c.ldg;
    a.out = c.out;
    a.ldo = c.ldo;
    return launch_attn_window_tc(ctx, a, st);
}

}  // namespace lbk

using namespace lbk;

namespace {

LatentShape shape_of(const lbk_latent_desc &d) {
    LatentShape s;
    s.heads = d.heads;
    s.dim = d.dim;
    s.rot_dim = d.rot_dim;
    s.vdim = d.vdim;
    s.kv_rank = d.kv_rank;
    s.q_rank = d.q_rank;
    return s;
}
Rotation rotation_of(const lbk_latent_desc &d) {
    Rotation r;
    r.freq = d.freq_dev;
    r.dims = static_cast<int>(d.rot_dim);
    r.factor = d.rot_factor;
    return r;
}
// parts of the work memory of one call, in 256-byte steps
struct LatentWork {
    size_t ql = 0, scratch = 0, ek = 0, ev = 0, zero = 0, total = 0, ecap = 0;
    LatentWork(const Ctx *ctx, int compute, const LatentShape &s, size_t rows, size_t cap, size_t length) {
        const size_t es = compute == LBK_COMPUTE_F32 ? 4 : 2;
        auto take = [&](size_t bytes) {
            const size_t at = total;
            total += (bytes + 255) / 256 * 256;
            return at;
        };
        if (length) {
            ecap = length;
            ek = take(s.heads * length * s.dp() * 2);
            ev = take(s.heads * length * s.vp() * 2);
            zero = take(4);
        } else {
            ql = take(rows * s.heads * s.pitch() * es);
            scratch = take(latent_scratch(ctx, rows, s, compute == LBK_COMPUTE_F32 ? 1 : latent_splits(cap)) * 4);
        }
    }
};

}  // namespace

extern "C" {

size_t lbk_latent_pitch(const lbk_latent_desc *d) { return d ? shape_of(*d).pitch() : 0; }
size_t lbk_latent_key_at(const lbk_latent_desc *d) { return d ? shape_of(*d).kvp() : 0; }
size_t lbk_latent_query_pitch(const lbk_latent_desc *d) { return d ? shape_of(*d).qp() : 0; }
size_t lbk_latent_query_rot_at(const lbk_latent_desc *d) { return d ? shape_of(*d).dp() : 0; }
int lbk_latent_expand_supported(const lbk_latent_desc *d) { return d && latent_expand_supported(shape_of(*d)) ? 1 : 0; }

int lbk_rotation_frequencies(size_t dims, double base, const double *yarn, double *freq_out, float *factor_out) {
    if (!freq_out || !factor_out || dims == 0 || dims % 2 || base <= 0.0) return fail(LBK_ERR_INVALID, "lbk_rotation_frequencies: an even number of dimensions and a positive base");
    YarnScaling y;
    if (yarn) {
        y.on = true;
        y.factor = yarn[0];
        y.original = yarn[1];
        y.fast = yarn[2];
        y.slow = yarn[3];
    }
    rotation_frequencies(dims, base, y, freq_out, factor_out);
    return LBK_OK;
}

int lbk_latent_prep(lbk_ctx *c, int compute, const lbk_latent_desc *d, const float *z_dev, size_t z_pitch, size_t rows, int rows_of_seq,
                    const int32_t *pos_dev, size_t cap, const float *q_norm_dev, const float *kv_norm_dev, float eps, void *cq_dev, size_t cq_pitch,
                    void *cache_dev, void *stream) {
    if (!c || !d) return fail(LBK_ERR_INVALID, "lbk_latent_prep: null argument");
    Ctx *ctx = reinterpret_cast<Ctx *>(c);
    LBK_CUDA(cudaSetDevice(ctx->device));
    LatentPrepCall p;
    p.compute = compute;
    p.s = shape_of(*d);
    p.z = z_dev;
    p.ldz = static_cast<long>(z_pitch);
    p.rows = rows;
    p.rows_of_seq = rows_of_seq;
    p.pos = pos_dev;
    p.cap = cap;
    p.q_norm = q_norm_dev;
    p.kv_norm = kv_norm_dev;
    p.eps = eps;
    p.rot = rotation_of(*d);
    p.cq = cq_dev;
    p.ldq = static_cast<long>(cq_pitch);
    p.cache = cache_dev;
    return launch_latent_prep(ctx, p, static_cast<cudaStream_t>(stream));
}

size_t lbk_latent_work_bytes(lbk_ctx *c, int compute, const lbk_latent_desc *d, size_t rows, size_t cap, size_t length) {
    return c && d ? LatentWork(reinterpret_cast<Ctx *>(c), compute, shape_of(*d), rows, cap, length).total : 0;
}

int lbk_latent_attn(lbk_ctx *c, int compute, const lbk_latent_desc *d, void *q_dev, size_t rows, int rows_of_seq, const int32_t *pos_dev, size_t cap,
                    const void *cache_dev, const uint16_t *ukv_dev, size_t ukv_pitch, float scale, const float *gate_dev, size_t gate_pitch, size_t length,
                    void *work_dev, void *out_dev, size_t out_pitch, void *stream) {
    if (!c || !d || !work_dev) return fail(LBK_ERR_INVALID, "lbk_latent_attn: null argument");
    if (ukv_pitch != dense_pitch(d->kv_rank)) return fail(LBK_ERR_SHAPE, "lbk_latent_attn: the weights' pitch is kv_rank rounded up to 64");
    Ctx *ctx = reinterpret_cast<Ctx *>(c);
    LBK_CUDA(cudaSetDevice(ctx->device));
    LatentAttnCall a;
    a.compute = compute;
    a.s = shape_of(*d);
    a.q = q_dev;
    a.rows = rows;
    a.rows_of_seq = rows_of_seq;
    a.pos = pos_dev;
    a.cap = cap;
    a.cache = cache_dev;
    const size_t kr = d->heads * d->dim, vr = d->heads * d->vdim;
    a.ukv = DenseWeight{ukv_dev, kr + vr, d->kv_rank, ukv_pitch};
    a.uk = DenseWeight{ukv_dev, kr, d->kv_rank, ukv_pitch};
    a.uv = DenseWeight{ukv_dev + kr * ukv_pitch, vr, d->kv_rank, ukv_pitch};
    a.scale = scale;
    a.rot = rotation_of(*d);
    a.gate = gate_dev;
    a.ldg = static_cast<long>(gate_pitch);
    a.out = out_dev;
    a.ldo = static_cast<long>(out_pitch);
    const LatentWork w(ctx, compute, a.s, rows, cap, length);
    char *base = static_cast<char *>(work_dev);
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (length) {
        a.length = length;
        a.ek = base + w.ek;
        a.ev = base + w.ev;
        a.ecap = w.ecap;
        a.zero = reinterpret_cast<int *>(base + w.zero);
        LBK_CUDA(cudaMemsetAsync(base, 0, w.total, st));  // the padding of keys and values has to hold numbers
        return launch_latent_expanded(ctx, a, st);
    }
    a.ql = base + w.ql;
    a.scratch = reinterpret_cast<float *>(base + w.scratch);
    a.splits = latent_splits(cap);
    return launch_latent_absorbed(ctx, a, st);
}

}  // extern "C"
