// Layer norm with a weight and no bias, (x - mean) / sqrt(var + eps) * w with var the mean of the squared
// deviations, or RMS norm, x / sqrt(mean(x^2) + eps) * w, and the "sandwich" step around a sublayer: the sublayer's output is normalised before it joins the
// f32 residual, and the next sublayer's input is the norm of the sum. One kernel does all of it for a row:
//
//     x += norm(y) * w_post        y: a projection's rows, or the outputs of a token's experts (gathered,
//                                  weighted and summed here) plus the gated shared expert
//     n  = norm(x) * w             to f32 (the head's input) and / or the compute type (a projection's input);
//                                  without w the sum itself (sublayers that read the residual un-normed)
//
// The row stays in registers between the four reductions (up to 8192 values at 256 threads a row; longer rows
// take 1024 threads).
#include "lbk_dense.cuh"
#include "lbk_dense_dev.cuh"
#include "lbk_ptx.cuh"

namespace lbk {

namespace {

struct NormParams {
    float *x;
    const float *y, *w_post, *w;
    MoeOut moe;
    int has_moe, n, rms;
    float eps;
    float *out_f;
    void *out_e;
    long lde;
};

template <int NT, int NV, typename T>
__global__ void __launch_bounds__(NT) sandwich_norm_kernel(const NormParams p) {
    ptx::pdl_trigger();
    ptx::pdl_wait();
    __shared__ float s_red[32];
    const int n = p.n;
    const size_t row = blockIdx.x;
    float *xr = p.x + row * n;
    float v[NV], u[NV];
    const float inv_n = 1.0f / static_cast<float>(n);
    const bool add = p.y || p.has_moe;
    if (add) {
        float s = 0.0f;
        float gate = 0.0f;
        if (p.has_moe && p.moe.shared) gate = dense::sigmoid(p.moe.gate[row * p.moe.ldg]);
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int i = threadIdx.x + j * NT;
            float t = 0.0f;
            if (i < n) {
                if (p.has_moe) {
                    for (int k = 0; k < p.moe.top; ++k) {
                        const int pl = p.moe.place[row * p.moe.top + k];
                        const float wk = p.moe.weight[row * p.moe.top + k];
                        t += wk * (p.moe.rows16 ? dense::bf16_f32(p.moe.rows16[static_cast<size_t>(pl) * p.moe.ld + i]) : p.moe.rows32[static_cast<size_t>(pl) * p.moe.ld + i]);
                    }
                    if (p.moe.shared) t += gate * p.moe.shared[row * n + i];
                } else {
                    t = p.y[row * n + i];
                }
                u[j] = xr[i];
            } else {
                u[j] = 0.0f;
            }
            v[j] = t;
            s += t;
        }
        const float mean = p.rms ? 0.0f : dense::block_sum<NT>(s, s_red) * inv_n;
        float ss = 0.0f;
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int i = threadIdx.x + j * NT;
            v[j] = i < n ? v[j] - mean : 0.0f;
            ss += v[j] * v[j];
        }
        const float r = 1.0f / sqrtf(dense::block_sum<NT>(ss, s_red) * inv_n + p.eps);
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int i = threadIdx.x + j * NT;
            if (i < n) {
                v[j] = u[j] + v[j] * r * p.w_post[i];
                xr[i] = v[j];
            }
        }
    } else {
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int i = threadIdx.x + j * NT;
            v[j] = i < n ? xr[i] : 0.0f;
        }
    }
    if (!p.w) {  // the sum itself
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int i = threadIdx.x + j * NT;
            if (i < n) {
                if (p.out_f) p.out_f[row * n + i] = v[j];
                if (p.out_e) dense::put(static_cast<T *>(p.out_e) + row * p.lde + i, v[j]);
            }
        }
        return;
    }
    float s = 0.0f;
#pragma unroll
    for (int j = 0; j < NV; ++j) s += v[j];
    const float mean = p.rms ? 0.0f : dense::block_sum<NT>(s, s_red) * inv_n;
    float ss = 0.0f;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
        const int i = threadIdx.x + j * NT;
        v[j] = i < n ? v[j] - mean : 0.0f;
        ss += v[j] * v[j];
    }
    const float r = 1.0f / sqrtf(dense::block_sum<NT>(ss, s_red) * inv_n + p.eps);
#pragma unroll
    for (int j = 0; j < NV; ++j) {
        const int i = threadIdx.x + j * NT;
        if (i < n) {
            const float o = v[j] * r * p.w[i];
            if (p.out_f) p.out_f[row * n + i] = o;
            if (p.out_e) dense::put(static_cast<T *>(p.out_e) + row * p.lde + i, o);
        }
    }
}

// The same with four neighbouring values a thread (rows of whole 16-byte units): the usual case.
template <int NV, typename T>
__global__ void __launch_bounds__(256) sandwich_norm_vec_kernel(const NormParams p) {
    ptx::pdl_trigger();
    ptx::pdl_wait();
    __shared__ float s_red[32];
    const int n = p.n, n4 = n >> 2;
    const size_t row = blockIdx.x;
    float4 *xr = reinterpret_cast<float4 *>(p.x + row * n);
    float4 v[NV];
    const float inv_n = 1.0f / static_cast<float>(n);
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    auto sum4 = [](const float4 &a) { return (a.x + a.y) + (a.z + a.w); };
    auto sq4 = [](const float4 &a) { return (a.x * a.x + a.y * a.y) + (a.z * a.z + a.w * a.w); };
    if (p.y || p.has_moe) {
        float4 u[NV];
        float s = 0.0f;
        float gate = 0.0f;
        if (p.has_moe && p.moe.shared) gate = dense::sigmoid(p.moe.gate[row * p.moe.ldg]);
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int i = threadIdx.x + j * 256;
            v[j] = u[j] = zero;
            if (i < n4) {
                u[j] = xr[i];
                if (!p.has_moe) {
                    v[j] = reinterpret_cast<const float4 *>(p.y + row * n)[i];
                } else if (p.moe.shared) {
                    const float4 a = reinterpret_cast<const float4 *>(p.moe.shared + row * n)[i];
                    v[j] = make_float4(gate * a.x, gate * a.y, gate * a.z, gate * a.w);
                }
            }
        }
        if (p.has_moe) {
            for (int k = 0; k < p.moe.top; ++k) {
                const size_t pl = p.moe.place[row * p.moe.top + k];
                const float wk = p.moe.weight[row * p.moe.top + k];
#pragma unroll
                for (int j = 0; j < NV; ++j) {
                    const int i = threadIdx.x + j * 256;
                    if (i < n4) {
                        float4 a;
                        if (p.moe.rows16) {
                            const uint2 b = reinterpret_cast<const uint2 *>(p.moe.rows16 + pl * p.moe.ld)[i];
                            a = make_float4(__uint_as_float(b.x << 16), __uint_as_float(b.x & 0xffff0000u), __uint_as_float(b.y << 16), __uint_as_float(b.y & 0xffff0000u));
                        } else {
                            a = reinterpret_cast<const float4 *>(p.moe.rows32 + pl * p.moe.ld)[i];
                        }
                        v[j].x += wk * a.x; v[j].y += wk * a.y; v[j].z += wk * a.z; v[j].w += wk * a.w;
                    }
                }
            }
        }
#pragma unroll
        for (int j = 0; j < NV; ++j) s += sum4(v[j]);
        const float mean = p.rms ? 0.0f : dense::block_sum<256>(s, s_red) * inv_n;
        float ss = 0.0f;
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int i = threadIdx.x + j * 256;
            v[j] = i < n4 ? make_float4(v[j].x - mean, v[j].y - mean, v[j].z - mean, v[j].w - mean) : zero;
            ss += sq4(v[j]);
        }
        const float r = 1.0f / sqrtf(dense::block_sum<256>(ss, s_red) * inv_n + p.eps);
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int i = threadIdx.x + j * 256;
            if (i < n4) {
                const float4 g = __ldg(reinterpret_cast<const float4 *>(p.w_post) + i);
                v[j] = make_float4(u[j].x + v[j].x * r * g.x, u[j].y + v[j].y * r * g.y, u[j].z + v[j].z * r * g.z, u[j].w + v[j].w * r * g.w);
                xr[i] = v[j];
            }
        }
    } else {
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int i = threadIdx.x + j * 256;
            v[j] = i < n4 ? xr[i] : zero;
        }
    }
    if (!p.w) {  // the sum itself
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int i = threadIdx.x + j * 256;
            if (i < n4) {
                if (p.out_f) reinterpret_cast<float4 *>(p.out_f + row * n)[i] = v[j];
                if (p.out_e) dense::put4(static_cast<T *>(p.out_e) + row * p.lde + 4 * i, v[j]);
            }
        }
        return;
    }
    float s = 0.0f;
#pragma unroll
    for (int j = 0; j < NV; ++j) s += sum4(v[j]);
    const float mean = p.rms ? 0.0f : dense::block_sum<256>(s, s_red) * inv_n;
    float ss = 0.0f;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
        const int i = threadIdx.x + j * 256;
        v[j] = i < n4 ? make_float4(v[j].x - mean, v[j].y - mean, v[j].z - mean, v[j].w - mean) : zero;
        ss += sq4(v[j]);
    }
    const float r = 1.0f / sqrtf(dense::block_sum<256>(ss, s_red) * inv_n + p.eps);
#pragma unroll
    for (int j = 0; j < NV; ++j) {
        const int i = threadIdx.x + j * 256;
        if (i < n4) {
            const float4 g = __ldg(reinterpret_cast<const float4 *>(p.w) + i);
            const float4 o = make_float4(v[j].x * r * g.x, v[j].y * r * g.y, v[j].z * r * g.z, v[j].w * r * g.w);
            if (p.out_f) reinterpret_cast<float4 *>(p.out_f + row * n)[i] = o;
            if (p.out_e) dense::put4(static_cast<T *>(p.out_e) + row * p.lde + 4 * i, o);
        }
    }
}

template <typename T>
int norm_impl(Ctx *ctx, const NormCall &c, cudaStream_t st) {
    if (c.rows == 0) return LBK_OK;
    if (!c.x || c.n == 0 || ((c.y || c.moe) && !c.w_post) || (c.w && !c.out_f && !c.out_e)) return fail(LBK_ERR_INVALID, "layer norm: null buffer or empty row");
    NormParams p{};
    p.x = c.x;
    p.y = c.y;
    p.w_post = c.w_post;
    p.w = c.w;
    if (c.moe) p.moe = *c.moe;
    p.has_moe = c.moe ? 1 : 0;
    p.n = static_cast<int>(c.n);
    p.rms = c.rms ? 1 : 0;
    p.eps = c.eps;
    p.out_f = c.out_f;
    p.out_e = c.out_e;
    p.lde = c.lde;
    const dim3 grid(static_cast<unsigned>(c.rows));
    uintptr_t bits = reinterpret_cast<uintptr_t>(c.x) | reinterpret_cast<uintptr_t>(c.y) | reinterpret_cast<uintptr_t>(c.w_post) |
                     reinterpret_cast<uintptr_t>(c.w) | reinterpret_cast<uintptr_t>(c.out_f) | reinterpret_cast<uintptr_t>(c.out_e);
    bool vec = c.n % 4 == 0 && c.n <= 8192 && c.lde % 4 == 0;
    if (c.moe) {
        bits |= reinterpret_cast<uintptr_t>(c.moe->rows16) | reinterpret_cast<uintptr_t>(c.moe->rows32) | reinterpret_cast<uintptr_t>(c.moe->shared);
        vec = vec && c.moe->ld % 4 == 0;
    }
    if (vec && (bits & 15) == 0) {
        if (c.n <= 1024) LBK_CUDA(launch_chained(sandwich_norm_vec_kernel<1, T>, grid, dim3(256), 0, st, p));
        else if (c.n <= 4096) LBK_CUDA(launch_chained(sandwich_norm_vec_kernel<4, T>, grid, dim3(256), 0, st, p));
        else LBK_CUDA(launch_chained(sandwich_norm_vec_kernel<8, T>, grid, dim3(256), 0, st, p));
    } else if (c.n <= 8192) {
        LBK_CUDA(launch_chained(sandwich_norm_kernel<256, 32, T>, grid, dim3(256), 0, st, p));
    } else if (c.n <= 32768) {
        LBK_CUDA(launch_chained(sandwich_norm_kernel<1024, 32, T>, grid, dim3(1024), 0, st, p));
    } else {
        return fail(LBK_ERR_UNSUPPORTED, "layer norm: rows of at most 32768 values (got %zu)", c.n);
    }
    LBK_CUDA(cudaGetLastError());
    ctx->launches++;
    return LBK_OK;
}

}  // namespace

int launch_sandwich_norm(Ctx *ctx, const NormCall &c, cudaStream_t st) {
    return c.compute == LBK_COMPUTE_F32 ? norm_impl<float>(ctx, c, st) : norm_impl<uint16_t>(ctx, c, st);
}

}  // namespace lbk

using namespace lbk;

static int sandwich_norm(lbk_ctx *c, bool rms, float *x_dev, const float *y_dev, const float *w_post_dev, const float *w_dev, size_t rows, size_t n,
                         float eps, float *out_f32_dev, uint16_t *out_bf16_dev, size_t out_bf16_pitch, void *stream) {
    if (!c) return fail(LBK_ERR_INVALID, "sandwich norm: context is null");
    Ctx *ctx = reinterpret_cast<Ctx *>(c);
    LBK_CUDA(cudaSetDevice(ctx->device));
    NormCall k;
    k.rms = rms;
    k.x = x_dev;
    k.y = y_dev;
    k.w_post = w_post_dev;
    k.w = w_dev;
    k.rows = rows;
    k.n = n;
    k.eps = eps;
    k.out_f = out_f32_dev;
    k.out_e = out_bf16_dev;
    k.lde = static_cast<long>(out_bf16_pitch);
    return launch_sandwich_norm(ctx, k, static_cast<cudaStream_t>(stream));
}

extern "C" int lbk_sandwich_norm(lbk_ctx *c, float *x_dev, const float *y_dev, const float *w_post_dev, const float *w_dev, size_t rows, size_t n,
                                 float eps, float *out_f32_dev, uint16_t *out_bf16_dev, size_t out_bf16_pitch, void *stream) {
    return sandwich_norm(c, false, x_dev, y_dev, w_post_dev, w_dev, rows, n, eps, out_f32_dev, out_bf16_dev, out_bf16_pitch, stream);
}

extern "C" int lbk_sandwich_rms_norm(lbk_ctx *c, float *x_dev, const float *y_dev, const float *w_post_dev, const float *w_dev, size_t rows, size_t n,
                                     float eps, float *out_f32_dev, uint16_t *out_bf16_dev, size_t out_bf16_pitch, void *stream) {
    return sandwich_norm(c, true, x_dev, y_dev, w_post_dev, w_dev, rows, n, eps, out_f32_dev, out_bf16_dev, out_bf16_pitch, stream);
}
