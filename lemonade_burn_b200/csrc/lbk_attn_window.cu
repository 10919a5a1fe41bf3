// Grouped-query attention under a sliding window with kept first tokens and a per-head distance bias: position i
// sees key j <= i when i - j < size or j < keep_first; the score is (q . k) * scale - slope_h * (i - j) with
// slope_h = 2^(-8 (h + 1) / heads); ordinary softmax. Window, kept tokens, scale, bias and head sizes are
// parameters (a window as long as the cache and no bias is plain causal attention).
//
// The keys a position sees are numbered without the gap: with lo = max(0, i - size + 1), the first
// min(keep_first, lo) of them are the kept tokens, the rest are lo .. i. Kernels walk these numbers, so nothing
// outside the window is read and kept tokens keep their true positions for the bias.
//
//   attn_window_decode_kernel  one new token per sequence, bf16: the query heads that share a KV head are the rows
//                              of one mma.sync tile (16 at a time), visible keys in slices of whole 64-key chunks,
//                              two stages of cp.async; scores, probabilities (two bf16 terms) and sums in f32.
//   attn_window_combine_kernel merges the slices.
//   attn_window_kernel         any head size up to 512 (f32: 1024), bf16 or f32, any rows: one block per (row, head). The
//                              32-bit path, portions of a few rows, and head sizes the others do not have.
// Prompt rows go to the tcgen05 kernel in lbk_attn_tc.cu.
#include "lbk_dense.cuh"
#include "lbk_dense_dev.cuh"
#include "lbk_ptx.cuh"

namespace lbk {

namespace {

struct WinParams {
    const void *q, *kc, *vc;
    const int *pos;
    int n, rows_of_seq, heads, kv_heads, dim, dimp, vdim, vdimp, cap, win, keep, splits;
    float scale, slope_unit;
    float *part;
    void *out;
    long ldo;
    int *err_word;
};

__device__ __forceinline__ float head_slope(const WinParams &p, int h) {
    return p.slope_unit == 0.0f ? 0.0f : p.slope_unit * exp2f(-8.0f * static_cast<float>(h + 1) / static_cast<float>(p.heads));
}
// the keys position `pos` sees, numbered 0 .. total - 1
struct Visible {
    int lo, kept, total;
    __device__ __forceinline__ Visible(const WinParams &p, int pos) {
        lo = max(0, pos - p.win + 1);
        kept = min(p.keep, lo);
        total = kept + pos - lo + 1;
    }
    __device__ __forceinline__ int key(int u) const { return u < kept ? u : lo + u - kept; }
};

// ---- any size, any type ---------------------------------------------------------------------------
template <typename T, int D>  // D: dimensions a lane holds (head sizes up to 32 * D)
__global__ void __launch_bounds__(128) attn_window_kernel(const WinParams p) {
    ptx::pdl_trigger();
    ptx::pdl_wait();
    __shared__ float s_m[4], s_l[4];
    __shared__ float s_acc[4][32 * D];
    const int head = blockIdx.x, row = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int seq = p.rows_of_seq >= 0 ? p.rows_of_seq : row;
    const int pos = p.rows_of_seq >= 0 ? p.pos[0] + row : p.pos[row];
    if (pos < 0 || pos >= p.cap) {
        if (tid == 0) atomicExch(p.err_word, 7);
        return;
    }
    const int kh = head / (p.heads / p.kv_heads);
    const T *q = static_cast<const T *>(p.q) + (static_cast<size_t>(row) * p.heads + head) * p.dimp;
    const T *kb = static_cast<const T *>(p.kc) + (static_cast<size_t>(seq) * p.kv_heads + kh) * p.cap * p.dimp;
    const T *vb = static_cast<const T *>(p.vc) + (static_cast<size_t>(seq) * p.kv_heads + kh) * p.cap * p.vdimp;
    const Visible vis(p, pos);
    const float slope = head_slope(p, head);
    float qv[D], acc[D];
#pragma unroll
    for (int i = 0; i < D; ++i) {
        const int d = lane + 32 * i;
        qv[i] = d < p.dim ? dense::get(q + d) : 0.0f;
        acc[i] = 0.0f;
    }
    float m = -INFINITY, l = 0.0f;
    constexpr int U = 4;  // keys in flight
    for (int u0 = warp * U; u0 < vis.total; u0 += 4 * U) {
        float s[U];
        int key[U];
#pragma unroll
        for (int j = 0; j < U; ++j) {
            key[j] = vis.key(min(u0 + j, vis.total - 1));
            const T *kr = kb + static_cast<size_t>(key[j]) * p.dimp;
            s[j] = 0.0f;
#pragma unroll
            for (int i = 0; i < D; ++i) {
                const int d = lane + 32 * i;
                if (d < p.dim) s[j] = fmaf(qv[i], dense::get(kr + d), s[j]);
            }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1)
#pragma unroll
            for (int j = 0; j < U; ++j) s[j] += __shfl_xor_sync(0xffffffffu, s[j], o);
        float nm = m;
#pragma unroll
        for (int j = 0; j < U; ++j) {
            s[j] = u0 + j < vis.total ? s[j] * p.scale - slope * static_cast<float>(pos - key[j]) : -INFINITY;
            nm = fmaxf(nm, s[j]);
        }
        const float corr = expf(m - nm);
        l *= corr;
#pragma unroll
        for (int i = 0; i < D; ++i) acc[i] *= corr;
#pragma unroll
        for (int j = 0; j < U; ++j) {
            const float w = expf(s[j] - nm);
            l += w;
            const T *vr = vb + static_cast<size_t>(key[j]) * p.vdimp;
#pragma unroll
            for (int i = 0; i < D; ++i) {
                const int d = lane + 32 * i;
                if (d < p.vdim) acc[i] = fmaf(w, dense::get(vr + d), acc[i]);
            }
        }
        m = nm;
    }
#pragma unroll
    for (int i = 0; i < D; ++i) s_acc[warp][lane + 32 * i] = acc[i];
    if (lane == 0) {
        s_m[warp] = m;
        s_l[warp] = l;
    }
    __syncthreads();
    const float gm = fmaxf(fmaxf(s_m[0], s_m[1]), fmaxf(s_m[2], s_m[3]));  // position i always sees itself: finite
    float wt[4], sum = 0.0f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
        wt[w] = s_m[w] == -INFINITY ? 0.0f : expf(s_m[w] - gm);
        sum += wt[w] * s_l[w];
    }
    T *o = static_cast<T *>(p.out) + static_cast<size_t>(row) * p.ldo + static_cast<size_t>(head) * p.vdim;
    for (int d = tid; d < p.vdim; d += 128)
        dense::put(o + d, (wt[0] * s_acc[0][d] + wt[1] * s_acc[1][d] + wt[2] * s_acc[2][d] + wt[3] * s_acc[3][d]) / sum);
}

// ---- decode on the tensor cores ---------------------------------------------------------------------
constexpr int kDwKeys = 64, kDwWarps = 4;
struct DwLayout {
    int krow, vrow, stage, q, total;  // bytes
    __host__ __device__ DwLayout(int dimp, int vdimp) {
        krow = dimp * 2 + 16;         // odd multiples of 16: eight rows start in different bank groups
        vrow = vdimp * 2 + 16;
        stage = kDwKeys * (krow + vrow);
        q = 2 * stage;
        total = q + 16 * krow + 32;
    }
};

// KS: 16-dimension steps of a key, VT: 8-dimension tiles of a value; upper bounds, or (EXACT) the sizes themselves
template <int KS, int VT, bool EXACT>
__global__ void __launch_bounds__(kDwWarps * 32) attn_window_decode_kernel(const WinParams p) {
    ptx::pdl_trigger();
    ptx::pdl_wait();
    extern __shared__ __align__(16) uint8_t dw_smem[];
    const int dimp = EXACT ? KS * 16 : p.dimp, vdimp = EXACT ? VT * 8 : p.vdimp;
    const DwLayout L(dimp, vdimp);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int group = p.heads / p.kv_heads, htiles = (group + 15) / 16;
    const int sp = blockIdx.x, kh = blockIdx.y / htiles, h0 = (blockIdx.y % htiles) * 16, b = blockIdx.z;
    const int nh = min(16, group - h0), head0 = kh * group + h0;  // this tile's query heads
    const int pos = p.pos[b];
    if (pos < 0 || pos >= p.cap) {
        if (tid == 0) atomicExch(p.err_word, 7);
        return;
    }
    const Visible vis(p, pos);
    const int per = ((vis.total + p.splits - 1) / p.splits + kDwKeys - 1) / kDwKeys * kDwKeys;
    const int u0 = min(vis.total, sp * per), u1 = min(vis.total, u0 + per);
    const uint16_t *kb = static_cast<const uint16_t *>(p.kc) + (static_cast<size_t>(b) * p.kv_heads + kh) * p.cap * dimp;
    const uint16_t *vb = static_cast<const uint16_t *>(p.vc) + (static_cast<size_t>(b) * p.kv_heads + kh) * p.cap * vdimp;
    const int ku = dimp / 8, vu = vdimp / 8;                  // 16-byte units per row
    for (int i = tid; i < 16 * ku; i += kDwWarps * 32) {
        const int r = i / ku, c = i - r * ku;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (r < nh) v = *reinterpret_cast<const uint4 *>(static_cast<const uint16_t *>(p.q) + (static_cast<size_t>(b) * p.heads + head0 + r) * dimp + c * 8);
        *reinterpret_cast<uint4 *>(dw_smem + L.q + r * L.krow + c * 16) = v;
    }
    auto stage = [&](int buf, int uc) {
        const int cnt = min(kDwKeys, u1 - uc);
        uint8_t *dk = dw_smem + buf * L.stage, *dv = dk + kDwKeys * L.krow;
        for (int i = tid; i < kDwKeys * (ku + vu); i += kDwWarps * 32) {
            const int r = i / (ku + vu), c = i - r * (ku + vu);
            uint8_t *dst = c < ku ? dk + r * L.krow + c * 16 : dv + r * L.vrow + (c - ku) * 16;
            if (r < cnt) {
                const int key = vis.key(uc + r);
                ptx::cp_async_16(ptx::smem_u32(dst), c < ku ? kb + static_cast<size_t>(key) * dimp + c * 8 : vb + static_cast<size_t>(key) * vdimp + (c - ku) * 8);
            } else {
                *reinterpret_cast<uint4 *>(dst) = make_uint4(0u, 0u, 0u, 0u);  // weight zero, but the bits must be numbers
            }
        }
        ptx::cp_async_commit();
    };
    const uint32_t s_q = ptx::smem_u32(dw_smem) + L.q + ((lane & 7) + 8 * ((lane >> 3) & 1)) * L.krow + (lane >> 4) * 16;
    const uint32_t k_lane0 = ptx::smem_u32(dw_smem) + (warp * 16 + (lane & 7)) * L.krow + (lane >> 3) * 16;
    const uint32_t v_lane0 = ptx::smem_u32(dw_smem) + kDwKeys * L.krow + (warp * 16 + (lane & 7) + 8 * ((lane >> 3) & 1)) * L.vrow + (lane >> 4) * 16;
    const float sl0 = head_slope(p, head0 + g), sl1 = head_slope(p, head0 + g + 8);
    const int ks_n = dimp / 16, vp_n = vdimp / 16;
    float o[VT][4];
#pragma unroll
    for (int j = 0; j < VT; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.0f;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.0f, l1 = 0.0f;
    if (u0 < u1) stage(0, u0);
    for (int uc = u0, it = 0; uc < u1; uc += kDwKeys, ++it) {
        if (it) __syncthreads();
        if (uc + kDwKeys < u1) {
            stage((it & 1) ^ 1, uc + kDwKeys);
            ptx::cp_async_wait<1>();
        } else {
            ptx::cp_async_wait<0>();
        }
        __syncthreads();
        const int w0 = uc + warp * 16;  // this warp's 16 keys
        if (w0 >= u1) continue;
        const uint32_t k_lane = k_lane0 + (it & 1) * L.stage, v_lane = v_lane0 + (it & 1) * L.stage;
        float s[2][4];
#pragma unroll
        for (int j = 0; j < 2; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.0f;
#pragma unroll
        for (int kp = 0; kp < KS / 2; ++kp) {  // 32 dimensions at a time; with an odd number of steps the last half is not used
            if (2 * kp < ks_n) {
                const bool both = 2 * kp + 1 < ks_n;
                uint32_t a0[4], a1[4];
                ptx::ldmatrix_x4(a0, s_q + kp * 64);
                if (both) ptx::ldmatrix_x4(a1, s_q + kp * 64 + 32);
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    uint32_t bb[4];
                    ptx::ldmatrix_x4(bb, k_lane + j * 8 * L.krow + kp * 64);
                    ptx::mma_bf16(s[j], a0, bb[0], bb[1]);
                    if (both) ptx::mma_bf16(s[j], a1, bb[2], bb[3]);
                }
            }
        }
        float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int u = w0 + 8 * j + 2 * t + e;
                const float dist = static_cast<float>(pos - vis.key(u));
                s[j][e] = u < u1 ? s[j][e] * p.scale - sl0 * dist : -INFINITY;
                s[j][2 + e] = u < u1 ? s[j][2 + e] * p.scale - sl1 * dist : -INFINITY;
                mx0 = fmaxf(mx0, s[j][e]);
                mx1 = fmaxf(mx1, s[j][2 + e]);
            }
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
        const float nm0 = fmaxf(m0, mx0), nm1 = fmaxf(m1, mx1);  // w0 < u1: at least one key is real, both are finite
        const float c0 = __expf(m0 - nm0), c1 = __expf(m1 - nm1);
        m0 = nm0;
        m1 = nm1;
        float ps0 = 0.0f, ps1 = 0.0f;
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const float e0 = __expf(s[j][0] - nm0), e1 = __expf(s[j][1] - nm0), e2 = __expf(s[j][2] - nm1), e3 = __expf(s[j][3] - nm1);
            ps0 += e0 + e1;
            ps1 += e2 + e3;
            ph[2 * j] = dense::bf16_pair(e0, e1);
            ph[2 * j + 1] = dense::bf16_pair(e2, e3);
            pl[2 * j] = dense::bf16_pair(e0 - __uint_as_float(ph[2 * j] << 16), e1 - __uint_as_float(ph[2 * j] & 0xffff0000u));
            pl[2 * j + 1] = dense::bf16_pair(e2 - __uint_as_float(ph[2 * j + 1] << 16), e3 - __uint_as_float(ph[2 * j + 1] & 0xffff0000u));
        }
        l0 = l0 * c0 + ps0;
        l1 = l1 * c1 + ps1;
#pragma unroll
        for (int j = 0; j < VT; ++j) {
            o[j][0] *= c0; o[j][1] *= c0;
            o[j][2] *= c1; o[j][3] *= c1;
        }
#pragma unroll
        for (int jp = 0; jp < VT / 2; ++jp)
            if (jp < vp_n) {
                uint32_t bb[4];
                ptx::ldmatrix_x4_trans(bb, v_lane + jp * 32);
                ptx::mma_bf16(o[2 * jp], ph, bb[0], bb[1]);
                ptx::mma_bf16(o[2 * jp], pl, bb[0], bb[1]);
                ptx::mma_bf16(o[2 * jp + 1], ph, bb[2], bb[3]);
                ptx::mma_bf16(o[2 * jp + 1], pl, bb[2], bb[3]);
            }
    }
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1);
    l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
    __syncthreads();  // the stages are free: [warp][16 heads][vdimp + 4] floats
    float *s_o = reinterpret_cast<float *>(dw_smem);
    const int mrow = vdimp + 4;
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        float *r = s_o + (warp * 16 + g + 8 * h) * mrow;
#pragma unroll
        for (int j = 0; j < VT; ++j)
            if (j < 2 * vp_n) *reinterpret_cast<float2 *>(r + 8 * j + 2 * t) = make_float2(o[j][2 * h], o[j][2 * h + 1]);
        if (t == 0) {
            r[vdimp] = h ? m1 : m0;
            r[vdimp + 1] = h ? l1 : l0;
        }
    }
    __syncthreads();
    const int prow = vdimp + 4;
    for (int i = tid; i < nh * (vdimp / 4); i += kDwWarps * 32) {
        const int r = i / (vdimp / 4), d = (i - r * (vdimp / 4)) * 4;
        float gm = -INFINITY;
#pragma unroll
        for (int w = 0; w < kDwWarps; ++w) gm = fmaxf(gm, s_o[(w * 16 + r) * mrow + vdimp]);
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
        float sum = 0.0f;
#pragma unroll
        for (int w = 0; w < kDwWarps; ++w) {
            const float *x = s_o + (w * 16 + r) * mrow;
            const float wm = x[vdimp];
            const float wt = wm == -INFINITY ? 0.0f : __expf(wm - gm);
            sum += wt * x[vdimp + 1];
            a.x += wt * x[d]; a.y += wt * x[d + 1]; a.z += wt * x[d + 2]; a.w += wt * x[d + 3];
        }
        if (p.splits == 1) {
            uint16_t *dst = static_cast<uint16_t *>(p.out) + static_cast<size_t>(b) * p.ldo + static_cast<size_t>(head0 + r) * p.vdim;
            const float v[4] = {a.x / sum, a.y / sum, a.z / sum, a.w / sum};
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (d + e < p.vdim) dst[d + e] = dense::f32_bf16(v[e]);
        } else {
            float *dst = p.part + ((static_cast<size_t>(b) * p.heads + head0 + r) * p.splits + sp) * prow;
            *reinterpret_cast<float4 *>(dst + d) = a;
            if (d == 0) {
                dst[vdimp] = gm;  // -inf for an empty slice: the merge gives it no weight
                dst[vdimp + 1] = sum;
            }
        }
    }
}

__global__ void __launch_bounds__(128) attn_window_combine_kernel(const WinParams p) {
    ptx::pdl_trigger();
    ptx::pdl_wait();
    extern __shared__ float s_w[];  // [splits]
    const int head = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, lane = tid & 31;
    const int prow = p.vdimp + 4;
    const float *part = p.part + (static_cast<size_t>(b) * p.heads + head) * p.splits * prow;
    // every warp works the weights out for itself (at most a few hundred slices)
    float mx = -INFINITY;
    for (int s = lane; s < p.splits; s += 32) mx = fmaxf(mx, part[static_cast<size_t>(s) * prow + p.vdimp]);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    float sum = 0.0f;
    for (int s = lane; s < p.splits; s += 32) {
        const float m = part[static_cast<size_t>(s) * prow + p.vdimp];
        const float w = m == -INFINITY ? 0.0f : __expf(m - mx);
        if (tid < 32) s_w[s] = w;
        sum += w * part[static_cast<size_t>(s) * prow + p.vdimp + 1];
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    __syncthreads();
    const float inv = 1.0f / sum;
    uint16_t *dst = static_cast<uint16_t *>(p.out) + static_cast<size_t>(b) * p.ldo + static_cast<size_t>(head) * p.vdim;
    for (int d = tid; d < p.vdim; d += 128) {
        float a = 0.0f;
#pragma unroll 8
        for (int s = 0; s < p.splits; ++s) a += s_w[s] * part[static_cast<size_t>(s) * prow + d];
        dst[d] = dense::f32_bf16(a * inv);
    }
}

constexpr size_t kMaxDim = 512, kMaxDim32 = 1024;  // 16-bit, 32-bit
constexpr size_t kTcMinRows = 8;  // prompt rows from which the 128-row tiles of the tcgen05 kernel are worth it

template <typename T>
int launch_generic(Ctx *ctx, const WinParams &p, cudaStream_t st) {
    const dim3 grid(static_cast<unsigned>(p.heads), static_cast<unsigned>(p.n));
    const int d = p.dim > p.vdim ? p.dim : p.vdim;
    if (d <= 128) LBK_CUDA(launch_chained(attn_window_kernel<T, 4>, grid, dim3(128), 0, st, p));
    else if (d <= 256) LBK_CUDA(launch_chained(attn_window_kernel<T, 8>, grid, dim3(128), 0, st, p));
    else if (d <= 512) LBK_CUDA(launch_chained(attn_window_kernel<T, 16>, grid, dim3(128), 0, st, p));
    else LBK_CUDA(launch_chained(attn_window_kernel<T, sizeof(T) == 4 ? 32 : 16>, grid, dim3(128), 0, st, p));
    LBK_CUDA(cudaGetLastError());
    ctx->launches++;
    return LBK_OK;
}

int attn_window_init(Ctx *) {
    const DwLayout small(64, 64), mid(128, 128), big(256, 256);
    LBK_CUDA(cudaFuncSetAttribute(attn_window_decode_kernel<4, 8, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, small.total));
    LBK_CUDA(cudaFuncSetAttribute(attn_window_decode_kernel<8, 16, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, mid.total));
    LBK_CUDA(cudaFuncSetAttribute(attn_window_decode_kernel<16, 32, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, big.total));
    LBK_CUDA(cudaFuncSetAttribute(attn_window_decode_kernel<4, 8, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, small.total));
    LBK_CUDA(cudaFuncSetAttribute(attn_window_decode_kernel<8, 16, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, mid.total));
    return LBK_OK;
}
const InitHook kInitAttnWindow(attn_window_init);

}  // namespace

// Slices for the longest run of keys a position of this cache can see: one 64-key chunk each, at most 64.
size_t attn_window_splits(size_t cap, const AttnMask &mask) {
    size_t most = cap;
    const size_t seen = static_cast<size_t>(mask.size) + static_cast<size_t>(mask.keep_first);
    if (seen < most) most = seen;
    const size_t s = (most + kDwKeys - 1) / kDwKeys;
    return s < 1 ? 1 : s > 64 ? 64 : s;
}
size_t attn_window_scratch(size_t b, size_t heads, size_t vdimp, size_t splits) { return b * heads * splits * (vdimp + 4); }

int launch_attn_window(Ctx *ctx, const AttnCall &c, cudaStream_t st) {
    if (c.n == 0) return LBK_OK;
    if (!c.q || !c.kc || !c.vc || !c.pos || !c.out) return fail(LBK_ERR_INVALID, "windowed attention: null buffer");
    if (c.kv_heads == 0 || c.heads % c.kv_heads || c.dim == 0 || c.vdim == 0 || c.dim > c.dimp || c.vdim > c.vdimp || c.dimp % 16 || c.vdimp % 16)
        return fail(LBK_ERR_SHAPE, "windowed attention: inconsistent head counts or sizes");
    const size_t most = c.compute == LBK_COMPUTE_F32 ? kMaxDim32 : kMaxDim;
    if (c.dim > most || c.vdim > most) return fail(LBK_ERR_UNSUPPORTED, "windowed attention: head sizes of at most %zu", most);
    if (c.n > 65535) return fail(LBK_ERR_UNSUPPORTED, "at most 65535 rows per call");
    WinParams p{};
    p.q = c.q;
    p.kc = c.kc;
    p.vc = c.vc;
    p.pos = c.pos;
    p.n = static_cast<int>(c.n);
    p.rows_of_seq = c.rows_of_seq;
    p.heads = static_cast<int>(c.heads);
    p.kv_heads = static_cast<int>(c.kv_heads);
    p.dim = static_cast<int>(c.dim);
    p.dimp = static_cast<int>(c.dimp);
    p.vdim = static_cast<int>(c.vdim);
    p.vdimp = static_cast<int>(c.vdimp);
    p.cap = static_cast<int>(c.cap);
    p.win = c.mask.size;
    p.keep = c.mask.keep_first;
    p.scale = c.scale;
    p.slope_unit = c.mask.alibi ? 1.0f : 0.0f;
    p.out = c.out;
    p.ldo = c.ldo;
    p.err_word = ctx->err_word;
    if (c.compute == LBK_COMPUTE_F32) return launch_generic<float>(ctx, p, st);
    const size_t dmax = c.dimp > c.vdimp ? c.dimp : c.vdimp;
    if (c.rows_of_seq >= 0) {
        if (c.n >= kTcMinRows && dmax <= 128) return launch_attn_window_tc(ctx, c, st);
        return launch_generic<uint16_t>(ctx, p, st);
    }
    if (dmax > 256) return launch_generic<uint16_t>(ctx, p, st);
    // slices: as many as the window has chunks, fewer when the batch alone fills the GPU (about four waves of
    // three blocks per SM)
    size_t splits = attn_window_splits(c.cap, c.mask);
    const size_t tiles = c.kv_heads * ((c.heads / c.kv_heads + 15) / 16);
    const size_t want = (12 * static_cast<size_t>(ctx->sm_count) + c.n * tiles - 1) / (c.n * tiles);
    if (want < splits) splits = want < 1 ? 1 : want;
    if (splits > 1 && !c.scratch) return fail(LBK_ERR_INVALID, "windowed attention: decode needs scratch memory");
    p.splits = static_cast<int>(splits);
    p.part = c.scratch;
    const dim3 grid(static_cast<unsigned>(splits), static_cast<unsigned>(tiles), static_cast<unsigned>(c.n));
    const size_t smem = static_cast<size_t>(DwLayout(p.dimp, p.vdimp).total);
    void (*k)(WinParams) = dmax <= 64 ? attn_window_decode_kernel<4, 8, false> : dmax <= 128 ? attn_window_decode_kernel<8, 16, false> : attn_window_decode_kernel<16, 32, false>;
    if (p.dimp == 64 && p.vdimp == 64) k = attn_window_decode_kernel<4, 8, true>;
    if (p.dimp == 128 && p.vdimp == 128) k = attn_window_decode_kernel<8, 16, true>;
    LBK_CUDA(launch_chained(k, grid, dim3(kDwWarps * 32), smem, st, p));
    LBK_CUDA(cudaGetLastError());
    ctx->launches++;
    if (splits > 1) {
        LBK_CUDA(launch_chained(attn_window_combine_kernel, dim3(static_cast<unsigned>(c.heads), static_cast<unsigned>(c.n)), dim3(128), splits * sizeof(float), st, p));
        LBK_CUDA(cudaGetLastError());
        ctx->launches++;
    }
    return LBK_OK;
}

}  // namespace lbk

using namespace lbk;

extern "C" size_t lbk_attn_window_scratch(size_t b, size_t heads, size_t vdim_pitch) { return attn_window_scratch(b, heads, vdim_pitch, 64); }

extern "C" int lbk_attn_window(lbk_ctx *c, int compute, const void *q_dev, const void *kcache_dev, const void *vcache_dev, const int32_t *pos_dev, size_t n,
                               int rows_of_seq, size_t heads, size_t kv_heads, size_t dim, size_t dim_pitch, size_t vdim, size_t vdim_pitch, size_t cap,
                               float scale, size_t window, size_t keep_first, int distance_bias, float *scratch_dev, void *out_dev, size_t out_pitch,
                               void *stream) {
    if (!c) return fail(LBK_ERR_INVALID, "lbk_attn_window: context is null");
    Ctx *ctx = reinterpret_cast<Ctx *>(c);
    LBK_CUDA(cudaSetDevice(ctx->device));
    AttnCall a;
    a.compute = compute;
    a.q = q_dev;
    a.kc = kcache_dev;
    a.vc = vcache_dev;
    a.pos = pos_dev;
    a.n = n;
    a.rows_of_seq = rows_of_seq;
    a.heads = heads;
    a.kv_heads = kv_heads;
    a.dim = dim;
    a.dimp = dim_pitch;
    a.vdim = vdim;
    a.vdimp = vdim_pitch;
    a.cap = cap;
    a.scale = scale;
    a.mask.size = window && window < (1u << 30) ? static_cast<int>(window) : 1 << 30;
    a.mask.keep_first = keep_first < (1u << 30) ? static_cast<int>(keep_first) : 1 << 30;
    a.mask.alibi = distance_bias != 0;
    a.scratch = scratch_dev;
    a.out = out_dev;
    a.ldo = static_cast<long>(out_pitch);
    return launch_attn_window(ctx, a, static_cast<cudaStream_t>(stream));
}
