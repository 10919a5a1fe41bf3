// Device helpers of the dense kernels: bf16 conversion, activations, block sums, and the epilogue that sends the
// value of (token, output row) where it belongs.
#pragma once

#include "lbk_dense.cuh"

namespace lbk {
namespace dense {

__device__ __forceinline__ float bf16_f32(uint16_t b) { return __uint_as_float(static_cast<uint32_t>(b) << 16); }
// two f32 -> one word of two bf16 (round to nearest even), `first` in the low half
__device__ __forceinline__ uint32_t bf16_pair(float first, float second) {
    uint32_t d;
    asm("cvt.rn.bf16x2.f32 %0, %1, %2;" : "=r"(d) : "f"(second), "f"(first));
    return d;
}
__device__ __forceinline__ uint16_t f32_bf16(float v) { return static_cast<uint16_t>(bf16_pair(v, 0.0f)); }

__device__ __forceinline__ void put(float *p, float v) { *p = v; }
__device__ __forceinline__ void put(uint16_t *p, float v) { *p = f32_bf16(v); }
__device__ __forceinline__ void put4(float *p, const float4 &v) { *reinterpret_cast<float4 *>(p) = v; }
__device__ __forceinline__ void put4(uint16_t *p, const float4 &v) {
    *reinterpret_cast<uint2 *>(p) = make_uint2(bf16_pair(v.x, v.y), bf16_pair(v.z, v.w));
}
__device__ __forceinline__ float get(const float *p) { return *p; }
__device__ __forceinline__ float get(const uint16_t *p) { return bf16_f32(*p); }

__device__ __forceinline__ float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
// 0.5 z (1 + tanh(u)) = z / (1 + e^(-2u)), u = sqrt(2/pi) (z + 0.044715 z^3)
template <bool EXACT>
__device__ __forceinline__ float gelu_tanh(float z) {
    const float u2 = 1.5957691216057308f * (z + 0.044715f * z * z * z);
    if (EXACT) return z / (1.0f + expf(-u2));
    return __fdividef(z, 1.0f + __expf(-u2));  // e^-u2 overflows to inf for large negative u: 0, as it should be
}
__device__ __forceinline__ float relu2(float z) {
    const float r = fmaxf(z, 0.0f);
    return r * r;
}

// z / (1 + e^-z); e^-z overflows to inf for large negative z: 0, as it should be
template <bool EXACT>
__device__ __forceinline__ float silu(float z) {
    if (EXACT) return z / (1.0f + expf(-z));
    return __fdividef(z, 1.0f + __expf(-z));
}

// Sum over the block; every thread gets it. `s_red`: 32 floats, may be reused right away.
template <int NT>
__device__ __forceinline__ float block_sum(float v, float *s_red) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) s_red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.0f;
#pragma unroll
    for (int w = 0; w < NT / 32; ++w) t += s_red[w];
    return t;
}

// Where output row r of a call goes, worked out once per row; the token is added per store.
struct RowPlan {
    int mode = 0;  // 0: drop, 1: f32, 2: compute type with squared relu, 3: compute type, 4: with silu
    float bias = 0.0f;
    char *base = nullptr;
    long stride = 0, seq_stride = 0;
    bool by_pos = false;
};
template <typename T>
__device__ __forceinline__ RowPlan row_plan(const DenseEpi &e, int r, int pos0) {
    RowPlan q;
    if (e.bias) q.bias = e.bias[r];
    if (e.kind == kEpiF32) {
        q.mode = 1;
        q.base = reinterpret_cast<char *>(static_cast<float *>(e.out) + r);
        q.stride = e.ld;
    } else if (e.kind == kEpiElem) {
        if (r >= e.f32_from) {
            q.mode = 1;
            q.base = reinterpret_cast<char *>(e.out2 + (r - e.f32_from));
            q.stride = e.ld2;
        } else {
            q.mode = r >= e.act_rows || e.act == kActNone ? 3 : e.act == kActRelu2 ? 2 : 4;
            q.base = reinterpret_cast<char *>(static_cast<T *>(e.out) + r);
            q.stride = e.ld;
        }
    } else {
        q.mode = 3;
        if (r < e.q_rows) {
            const int h = r / e.dim, d = r - h * e.dim;
            q.base = reinterpret_cast<char *>(static_cast<T *>(e.out) + h * e.dimp + d + (d >= e.q_split ? e.q_gap : 0));
            q.stride = e.ld;
        } else {
            const bool is_k = r < e.q_rows + e.k_rows;
            const int rr = r - e.q_rows - (is_k ? 0 : e.k_rows), dd = is_k ? e.dim : e.vdim, dp = is_k ? e.dimp : e.vdimp;
            const int h = rr / dd, d = rr - h * dd;
            T *c = static_cast<T *>(is_k ? e.kc : e.vc);
            if (e.rows_of_seq >= 0) {
                q.base = reinterpret_cast<char *>(c + ((static_cast<size_t>(e.rows_of_seq) * e.kv_heads + h) * e.cap + pos0) * dp + d);
                q.stride = dp;
            } else {
                q.base = reinterpret_cast<char *>(c + static_cast<size_t>(h) * e.cap * dp + d);
                q.stride = dp;
                q.seq_stride = static_cast<long>(e.kv_heads) * e.cap * dp;
                q.by_pos = true;
            }
        }
    }
    return q;
}
template <typename T>
__device__ __forceinline__ void row_store(const DenseEpi &e, const RowPlan &q, int t, float v) {
    long off = static_cast<long>(t) * q.stride;
    if (q.by_pos) {
        const int pos = e.pos[t];
        if (pos < 0 || pos >= e.cap) {
            atomicExch(e.err_word, 7);
            return;
        }
        off = static_cast<long>(t) * q.seq_stride + static_cast<long>(pos) * q.stride;
    }
    v += q.bias;
    if (q.mode == 1) reinterpret_cast<float *>(q.base)[off] = v;
    else if (q.mode) put(reinterpret_cast<T *>(q.base) + off, q.mode == 3 ? v : q.mode == 2 ? relu2(v) : silu<sizeof(T) == 4>(v));
}
// Tokens t0 .. t0 + min(N, cnt) - 1 of one row at once, the choice of what to do with them outside the loop.
template <typename T, int N>
__device__ __forceinline__ void row_store_run(const DenseEpi &e, const RowPlan &q, int t0, int cnt, const uint32_t (&v)[N]) {
    if (q.mode == 0) return;
    if (q.by_pos) {
#pragma unroll
        for (int i = 0; i < N; ++i)
            if (i < cnt) row_store<T>(e, q, t0 + i, __uint_as_float(v[i]));
        return;
    }
    const long first = static_cast<long>(t0) * q.stride;
    if (q.mode == 1) {
        float *o = reinterpret_cast<float *>(q.base) + first;
#pragma unroll
        for (int i = 0; i < N; ++i)
            if (i < cnt) o[i * q.stride] = __uint_as_float(v[i]) + q.bias;
        return;
    }
    T *o = reinterpret_cast<T *>(q.base) + first;
    if (q.mode == 2) {
#pragma unroll
        for (int i = 0; i < N; ++i)
            if (i < cnt) put(o + i * q.stride, relu2(__uint_as_float(v[i]) + q.bias));
    } else if (q.mode == 4) {
#pragma unroll
        for (int i = 0; i < N; ++i)
            if (i < cnt) put(o + i * q.stride, silu<sizeof(T) == 4>(__uint_as_float(v[i]) + q.bias));
    } else {
#pragma unroll
        for (int i = 0; i < N; ++i)
            if (i < cnt) put(o + i * q.stride, __uint_as_float(v[i]) + q.bias);
    }
}
// A prompt pass whose positions do not fit the cache must not store anything.
__device__ __forceinline__ bool rows_fit(const DenseEpi &e, int m, int &pos0) {
    pos0 = 0;
    if (e.kind != kEpiQkv || e.rows_of_seq < 0) return true;
    pos0 = *e.pos;
    if (pos0 >= 0 && pos0 + m <= e.cap) return true;
    if (threadIdx.x == 0) atomicExch(e.err_word, 7);
    return false;
}

}  // namespace dense
}  // namespace lbk
