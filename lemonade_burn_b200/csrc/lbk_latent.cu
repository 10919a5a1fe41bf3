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
//   latent_absorb_kernel  W_uk,h^T q and the rotated part: a query against cache rows
//   latent_attn_kernel    bf16: 16 or 32 heads x 64 positions at a time on mma.sync, the positions' rows staged once by
//                         cp.async for both products; scores, softmax and sums f32, probabilities in two bf16 terms.
//                         Slices of the positions over the blocks of the grid.
//   latent_out_kernel     merges the slices, W_uv,h, the head's gate
#include <algorithm>
#include <cmath>

#include "lbk_dense_dev.cuh"
#include "lbk_mixers.cuh"
#include "lbk_ptx.cuh"

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

// One block: head blockIdx.x, 128 latent dimensions, four tokens. Threads: 16 groups of 8 dimensions x 16 shares of the
// head's unrotated dimensions.
constexpr int kAbsCols = 128, kAbsTok = 4;
template <typename T>
__global__ void __launch_bounds__(256) latent_absorb_kernel(const QueryParams p) {
    ptx::pdl_trigger();
    ptx::pdl_wait();
    extern __shared__ float s_q[];                       // [kAbsTok][dim]
    __shared__ float s_part[8][kAbsTok][kAbsCols];
    const int h = blockIdx.x, c0 = blockIdx.y * kAbsCols, t0 = blockIdx.z * kAbsTok, tid = threadIdx.x;
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

// ---- attention over the latents, bf16 ---------------------------------------------------------------
constexpr int kLKeys = 64, kLWarps = 8;
constexpr int kLValues = 4;         // 16-dimension tiles of the latent a warp accumulates: latents of up to 512
struct LatentLayout {
    int krow, prow, q, ph, pl, mx, total;  // bytes
    __host__ __device__ LatentLayout(int width, int mt) {
        krow = width * 2 + 16;             // an odd multiple of 16: eight rows start in different bank groups
        prow = kLKeys * 2 + 16;
        q = 2 * kLKeys * krow;
        ph = q + 16 * mt * krow;
        pl = ph + 16 * mt * prow;
        mx = pl + 16 * mt * prow;
        total = mx + 2 * kLWarps * 16 * mt * 4;
    }
};
struct LatentParams {
    const uint16_t *ql, *cache;
    const int *pos;
    int rows_of_seq, heads, width, kvp, pitch, cap, splits;
    float scale;
    float *part;                    // [row][head][split][kvp + 4]
    int *err_word;
};

template <int MT>  // tiles of 16 heads a block takes
__global__ void __launch_bounds__(kLWarps * 32) latent_attn_kernel(const LatentParams p) {
    ptx::pdl_trigger();
    ptx::pdl_wait();
    extern __shared__ __align__(16) uint8_t la_smem[];
    const LatentLayout L(p.width, MT);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int sp = blockIdx.x, h0 = blockIdx.y * 16 * MT, row = blockIdx.z, nh = min(16 * MT, p.heads - h0);
    const int seq = p.rows_of_seq >= 0 ? p.rows_of_seq : row, pos = p.rows_of_seq >= 0 ? p.pos[0] + row : p.pos[row];
    if (pos < 0 || pos >= p.cap) {
        if (tid == 0) atomicExch(p.err_word, 7);
        return;
    }
    const int total = pos + 1, per = ((total + p.splits - 1) / p.splits + kLKeys - 1) / kLKeys * kLKeys;
    const int u0 = min(total, sp * per), u1 = min(total, u0 + per);
    const uint16_t *kb = p.cache + static_cast<size_t>(seq) * p.cap * p.pitch;
    const int ku = p.width / 8;                              // 16-byte units of a row
    const uint32_t sm = ptx::smem_u32(la_smem);
    for (int i = tid; i < 16 * MT * ku; i += kLWarps * 32) {
        const int r = i / ku, c = i - r * ku;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (r < nh) v = *reinterpret_cast<const uint4 *>(p.ql + (static_cast<size_t>(row) * p.heads + h0 + r) * p.pitch + c * 8);
        *reinterpret_cast<uint4 *>(la_smem + L.q + r * L.krow + c * 16) = v;
    }
    auto stage = [&](int buf, int uc) {
        const int cnt = min(kLKeys, u1 - uc);
        for (int i = tid; i < kLKeys * ku; i += kLWarps * 32) {
            const int r = i / ku, c = i - r * ku;
            uint8_t *dst = la_smem + (buf * kLKeys + r) * L.krow + c * 16;
            if (r < cnt) ptx::cp_async_16(ptx::smem_u32(dst), kb + static_cast<size_t>(uc + r) * p.pitch + c * 8);
            else *reinterpret_cast<uint4 *>(dst) = make_uint4(0u, 0u, 0u, 0u);  // weight zero, but the bits must be numbers
        }
        ptx::cp_async_commit();
    };
    float *s_mx = reinterpret_cast<float *>(la_smem + L.mx);  // [warp][16 MT], then the same for the sums
    const uint32_t q_lane = sm + L.q + ((lane & 7) + 8 * ((lane >> 3) & 1)) * L.krow + (lane >> 4) * 16;
    const uint32_t k_lane0 = sm + (warp * 8 + (lane & 7)) * L.krow + (lane >> 3) * 16;
    const uint32_t v_lane0 = sm + ((lane & 7) + 8 * ((lane >> 3) & 1)) * L.krow + (lane >> 4) * 16;
    const uint32_t p_lane = sm + ((lane & 7) + 8 * ((lane >> 3) & 1)) * L.prow + (lane >> 4) * 16;
    const int ksteps = p.width / 16, vtiles = p.kvp / 16;
    float o[MT][kLValues][2][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int i = 0; i < kLValues; ++i)
#pragma unroll
            for (int e = 0; e < 2; ++e) o[m][i][e][0] = o[m][i][e][1] = o[m][i][e][2] = o[m][i][e][3] = 0.0f;
    float mrow[MT][2], lrow[MT][2];
#pragma unroll
    for (int m = 0; m < MT; ++m) mrow[m][0] = mrow[m][1] = -INFINITY, lrow[m][0] = lrow[m][1] = 0.0f;
    if (u0 < u1) stage(0, u0);
    for (int uc = u0, it = 0; uc < u1; uc += kLKeys, ++it) {
        if (it) __syncthreads();                             // the other buffer and the probabilities have been read
        if (uc + kLKeys < u1) {
            stage((it & 1) ^ 1, uc + kLKeys);
            ptx::cp_async_wait<1>();
        } else {
            ptx::cp_async_wait<0>();
        }
        __syncthreads();
        const uint32_t boff = (it & 1) * kLKeys * L.krow;
        float s[MT][4];
#pragma unroll
        for (int m = 0; m < MT; ++m) s[m][0] = s[m][1] = s[m][2] = s[m][3] = 0.0f;
#pragma unroll 2
        for (int kp = 0; kp < ksteps; kp += 2) {             // 32 dimensions; with an odd number of steps the last half is not used
            uint32_t bb[4];
            ptx::ldmatrix_x4(bb, k_lane0 + boff + kp * 32);
#pragma unroll
            for (int m = 0; m < MT; ++m) {
                uint32_t a[4];
                ptx::ldmatrix_x4(a, q_lane + m * 16 * L.krow + kp * 32);
                ptx::mma_bf16(s[m], a, bb[0], bb[1]);
            }
            if (kp + 1 < ksteps) {
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    uint32_t a[4];
                    ptx::ldmatrix_x4(a, q_lane + m * 16 * L.krow + kp * 32 + 32);
                    ptx::mma_bf16(s[m], a, bb[2], bb[3]);
                }
            }
        }
        const int key = uc + warp * 8 + 2 * t;               // this lane's keys: key, key + 1
#pragma unroll
        for (int m = 0; m < MT; ++m) {
#pragma unroll
            for (int e = 0; e < 4; ++e) s[m][e] = key + (e & 1) < u1 ? s[m][e] * p.scale : -INFINITY;
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                float mx = fmaxf(s[m][2 * r], s[m][2 * r + 1]);
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
                if (t == 0) s_mx[warp * 16 * MT + m * 16 + g + 8 * r] = mx;
            }
        }
        __syncthreads();
        float corr[MT][2];
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                float nm = mrow[m][r];
#pragma unroll
                for (int w = 0; w < kLWarps; ++w) nm = fmaxf(nm, s_mx[w * 16 * MT + m * 16 + g + 8 * r]);
                corr[m][r] = __expf(mrow[m][r] - nm);        // nm is finite: a chunk has at least one key
                mrow[m][r] = nm;
                const float e0 = __expf(s[m][2 * r] - nm), e1 = __expf(s[m][2 * r + 1] - nm);
                lrow[m][r] = lrow[m][r] * corr[m][r] + e0 + e1;
                const uint32_t hi = dense::bf16_pair(e0, e1);
                const uint32_t lo = dense::bf16_pair(e0 - __uint_as_float(hi << 16), e1 - __uint_as_float(hi & 0xffff0000u));
                const int at = (m * 16 + g + 8 * r) * L.prow + (warp * 8 + 2 * t) * 2;
                *reinterpret_cast<uint32_t *>(la_smem + L.ph + at) = hi;
                *reinterpret_cast<uint32_t *>(la_smem + L.pl + at) = lo;
            }
        __syncthreads();
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int i = 0; i < kLValues; ++i)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    o[m][i][e][0] *= corr[m][0]; o[m][i][e][1] *= corr[m][0];
                    o[m][i][e][2] *= corr[m][1]; o[m][i][e][3] *= corr[m][1];
                }
#pragma unroll
        for (int ks = 0; ks < kLKeys / 16; ++ks) {
            uint32_t ph[MT][4], pl[MT][4];
#pragma unroll
            for (int m = 0; m < MT; ++m) {
                ptx::ldmatrix_x4(ph[m], p_lane + L.ph + m * 16 * L.prow + ks * 32);
                ptx::ldmatrix_x4(pl[m], p_lane + L.pl + m * 16 * L.prow + ks * 32);
            }
#pragma unroll
            for (int i = 0; i < kLValues; ++i) {
                const int vt = warp + kLWarps * i;
                if (vt < vtiles) {
                    uint32_t bb[4];
                    ptx::ldmatrix_x4_trans(bb, v_lane0 + boff + ks * 16 * L.krow + vt * 32);
#pragma unroll
                    for (int m = 0; m < MT; ++m) {
                        ptx::mma_bf16(o[m][i][0], ph[m], bb[0], bb[1]);
                        ptx::mma_bf16(o[m][i][0], pl[m], bb[0], bb[1]);
                        ptx::mma_bf16(o[m][i][1], ph[m], bb[2], bb[3]);
                        ptx::mma_bf16(o[m][i][1], pl[m], bb[2], bb[3]);
                    }
                }
            }
        }
    }
    // this slice's sums and, unscaled, the weighted latents
    float *s_l = s_mx + kLWarps * 16 * MT;
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            float v = lrow[m][r];
            v += __shfl_xor_sync(0xffffffffu, v, 1);
            v += __shfl_xor_sync(0xffffffffu, v, 2);
            if (t == 0) s_l[warp * 16 * MT + m * 16 + g + 8 * r] = v;
        }
    __syncthreads();
    const int prow = p.kvp + 4;
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int hr = m * 16 + g + 8 * r;
            if (hr >= nh) continue;
            float *dst = p.part + ((static_cast<size_t>(row) * p.heads + h0 + hr) * p.splits + sp) * prow;
#pragma unroll
            for (int i = 0; i < kLValues; ++i) {
                const int vt = warp + kLWarps * i;
                if (vt < vtiles)
#pragma unroll
                    for (int e = 0; e < 2; ++e) *reinterpret_cast<float2 *>(dst + vt * 16 + e * 8 + 2 * t) = make_float2(o[m][i][e][2 * r], o[m][i][e][2 * r + 1]);
            }
            if (warp == 0 && t == 0) {
                float sum = 0.0f;
#pragma unroll
                for (int w = 0; w < kLWarps; ++w) sum += s_l[w * 16 * MT + hr];
                dst[p.kvp] = mrow[m][r];                     // -inf for an empty slice: the merge gives it no weight
                dst[p.kvp + 1] = sum;
            }
        }
}

// ---- out: merge, W_uv, gate -----------------------------------------------------------------------------
struct OutParams {
    const float *part;              // slices, or (splits = 0) the weighted latents themselves, [row][heads][kv_rank]
    int rows, heads, splits, vdim, kv_rank, kvp;
    const uint16_t *uv;
    int uv_pitch;
    const float *gate;
    long ldg, ldo;
    void *out;
};
constexpr int kOutTok = 4, kOutRows = 32;
template <typename T>
__global__ void __launch_bounds__(256) latent_out_kernel(const OutParams p) {
    ptx::pdl_trigger();
    ptx::pdl_wait();
    extern __shared__ float s_dyn[];                         // [kOutTok][uv_pitch], [splits] weights
    __shared__ float4 s_half[128];                           // the second half of the slices' sum (latents of up to 512)
    float *s_w = s_dyn + kOutTok * p.uv_pitch;
    const int h = blockIdx.x, e0 = blockIdx.y * kOutRows, t0 = blockIdx.z * kOutTok, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int toks = min(kOutTok, p.rows - t0);
    for (int t = 0; t < kOutTok; ++t) {
        float *x = s_dyn + t * p.uv_pitch;
        if (t >= toks) {
            for (int i = tid; i < p.uv_pitch; i += 256) x[i] = 0.0f;
            continue;
        }
        const size_t rh = static_cast<size_t>(t0 + t) * p.heads + h;
        if (p.splits == 0) {
            for (int i = tid; i < p.uv_pitch; i += 256) x[i] = i < p.kv_rank ? p.part[rh * p.kv_rank + i] : 0.0f;
            continue;
        }
        const int prow = p.kvp + 4;
        const float *part = p.part + rh * p.splits * prow;
        // every warp works the weights out for itself
        float mx = -INFINITY, sum = 0.0f;
        for (int s = lane; s < p.splits; s += 32) mx = fmaxf(mx, part[static_cast<size_t>(s) * prow + p.kvp]);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        __syncthreads();                                     // the weights of the token before have been read
        for (int s = lane; s < p.splits; s += 32) {
            const float m = part[static_cast<size_t>(s) * prow + p.kvp];
            const float w = m == -INFINITY ? 0.0f : __expf(m - mx);
            if (warp == 0) s_w[s] = w;
            sum += w * part[static_cast<size_t>(s) * prow + p.kvp + 1];
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        __syncthreads();
        const float inv = 1.0f / sum;
        // four values a thread, every second slice; what lies between kv_rank and kvp is zero
        const int i = (tid & 127) * 4, half = tid >> 7;
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < p.kvp) {
#pragma unroll 16
            for (int s = half; s < p.splits; s += 2) {
                const float4 v = *reinterpret_cast<const float4 *>(part + static_cast<size_t>(s) * prow + i);
                const float w = s_w[s];
                a.x = fmaf(w, v.x, a.x); a.y = fmaf(w, v.y, a.y); a.z = fmaf(w, v.z, a.z); a.w = fmaf(w, v.w, a.w);
            }
        }
        if (half) s_half[tid & 127] = a;
        __syncthreads();
        if (!half && i < p.uv_pitch) {
            const float4 b = s_half[tid];
            *reinterpret_cast<float4 *>(x + i) = make_float4((a.x + b.x) * inv, (a.y + b.y) * inv, (a.z + b.z) * inv, (a.w + b.w) * inv);
        }
    }
    __syncthreads();
    for (int r = warp; r < kOutRows; r += 8) {
        const int e = e0 + r;
        if (e >= p.vdim) break;
        const uint16_t *w = p.uv + static_cast<size_t>(h * p.vdim + e) * p.uv_pitch;
        float acc[kOutTok] = {};
        for (int i = lane * 8; i < p.uv_pitch; i += 256) {
            const uint4 v = *reinterpret_cast<const uint4 *>(w + i);
            const uint32_t wv[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
            for (int t = 0; t < kOutTok; ++t) {
                const float4 a = *reinterpret_cast<const float4 *>(s_dyn + t * p.uv_pitch + i), b = *reinterpret_cast<const float4 *>(s_dyn + t * p.uv_pitch + i + 4);
                const float x[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    acc[t] = fmaf(__uint_as_float(wv[k] << 16), x[2 * k], acc[t]);
                    acc[t] = fmaf(__uint_as_float(wv[k] & 0xffff0000u), x[2 * k + 1], acc[t]);
                }
            }
        }
#pragma unroll
        for (int t = 0; t < kOutTok; ++t) {
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) acc[t] += __shfl_xor_sync(0xffffffffu, acc[t], o);
            if (lane == 0 && t < toks)
                dense::put(static_cast<T *>(p.out) + static_cast<size_t>(t0 + t) * p.ldo + static_cast<size_t>(h) * p.vdim + e,
                           acc[t] * dense::sigmoid(p.gate[static_cast<size_t>(t0 + t) * p.ldg + h]));
        }
    }
}

constexpr size_t kMaxSplits = 64;
constexpr int kLatentSmem = 227 * 1024;

bool latent_mma_supported(const LatentShape &s) {
    return s.kvp() <= kLWarps * kLValues * 16 && LatentLayout(static_cast<int>(s.kvp() + s.rp()), 1).total <= kLatentSmem;
}

int latent_init(Ctx *ctx) {
    const int most = static_cast<int>(ctx->smem_optin) < kLatentSmem ? static_cast<int>(ctx->smem_optin) : kLatentSmem;
    LBK_CUDA(cudaFuncSetAttribute(latent_attn_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, most));
    LBK_CUDA(cudaFuncSetAttribute(latent_attn_kernel<2>, cudaFuncAttributeMaxDynamicSharedMemorySize, most));
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
    const dim3 agrid(static_cast<unsigned>(c.s.heads), static_cast<unsigned>((c.s.kvp() + kAbsCols - 1) / kAbsCols), static_cast<unsigned>((c.rows + kAbsTok - 1) / kAbsTok));
    LBK_CUDA(launch_chained(f32 ? latent_absorb_kernel<float> : latent_absorb_kernel<uint16_t>, agrid, dim3(256), kAbsTok * c.s.dim * sizeof(float), st, qp));
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
        if (!latent_mma_supported(c.s)) return fail(LBK_ERR_UNSUPPORTED, "latent attention in bf16: latents of at most 512 values");
        LatentParams p{};
        p.ql = static_cast<const uint16_t *>(c.ql);
        p.cache = static_cast<const uint16_t *>(c.cache);
        p.pos = c.pos;
        p.rows_of_seq = c.rows_of_seq;
        p.heads = qp.heads;
        p.width = static_cast<int>(c.s.kvp() + c.s.rp());
        p.kvp = qp.kvp;
        p.pitch = qp.pitch;
        p.cap = static_cast<int>(c.cap);
        p.scale = c.scale;
        p.part = c.scratch;
        p.err_word = ctx->err_word;
        const bool two = c.s.heads > 16 && LatentLayout(p.width, 2).total <= kLatentSmem;
        const size_t tiles = (c.s.heads + (two ? 31 : 15)) / (two ? 32 : 16);
        // about one block per SM: as many slices as that leaves
        const size_t want = static_cast<size_t>(ctx->sm_count) / (c.rows * tiles);
        p.splits = static_cast<int>(want < 1 ? 1 : want < c.splits ? want : c.splits);
        op.splits = p.splits;
        const dim3 grid(static_cast<unsigned>(p.splits), static_cast<unsigned>(tiles), static_cast<unsigned>(c.rows));
        LBK_CUDA(launch_chained(two ? latent_attn_kernel<2> : latent_attn_kernel<1>, grid, dim3(kLWarps * 32), static_cast<size_t>(LatentLayout(p.width, two ? 2 : 1).total), st, p));
        LBK_CUDA(cudaGetLastError());
        ctx->launches++;
    }
    const dim3 ogrid(static_cast<unsigned>(c.s.heads), static_cast<unsigned>((c.s.vdim + kOutRows - 1) / kOutRows), static_cast<unsigned>((c.rows + kOutTok - 1) / kOutTok));
    LBK_CUDA(launch_chained(f32 ? latent_out_kernel<float> : latent_out_kernel<uint16_t>, ogrid, dim3(256), (kOutTok * c.uv.pitch + kMaxSplits) * sizeof(float), st, op));
    LBK_CUDA(cudaGetLastError());
    ctx->launches++;
    return LBK_OK;
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
