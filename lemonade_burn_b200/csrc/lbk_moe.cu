// Mixture of experts: routing and the few-token expert kernels.
//
// Router: z = W_router h (rows of a projection, f32), s = softmax(z) over all experts, the `top` largest are chosen
// (the lower index first among equals) and their s are the weights, not renormalised. Expert: down(relu2(up h)).
// A shared expert of the same form runs for every token, times the sigmoid of one gate logit per token.
//
//   moe_topk / moe_scan / moe_scatter   prompt passes: chosen experts and weights, expert offsets, the tokens' rows
//                    copied in expert order; the expert projections are then dense_gemm_kernel / dense_f32_kernel
//                    calls over the sorted rows (lbk_dense.cu), and the norm behind the layer gathers, weights and sums
//                    each token's rows (lbk_layernorm.cu).
//   moe_few_up_kernel, moe_few_down_kernel   up to 16 tokens, bf16. Bound: HBM, the chosen experts' weights once.
//                    A persistent CTA routes the tokens itself, takes (chosen expert, 16 rows) units, and folds
//                    the routing weight into the activation. The down kernel owns 16 output rows and walks the
//                    shared and all chosen experts' columns as one long K, so no partial sums leave the CTA and
//                    the result does not depend on any order of arrival.
#include "lbk_dense.cuh"
#include "lbk_dense_dev.cuh"
#include "lbk_ptx.cuh"

namespace lbk {

namespace {

constexpr int kMaxTop = 32;
constexpr int kMaxExperts = 1024;

// One warp routes one token: softmax over E logits, then `top` rounds of "largest that is left". Lane l holds
// experts l, l + 32, ... Calls put(k, expert, weight) in every lane.
template <int R, typename F>
__device__ __forceinline__ void route_token(const float *z, int E, int top, int lane, F put) {
    float v[R];
    float mx = -INFINITY;
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int e = lane + 32 * i;
        v[i] = e < E ? z[e] : -INFINITY;
        mx = fmaxf(mx, v[i]);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    float sum = 0.0f;
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int e = lane + 32 * i;
        v[i] = e < E ? expf(v[i] - mx) : -1.0f;
        if (e < E) sum += v[i];
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    for (int k = 0; k < top; ++k) {
        float bv = -1.0f;
        int be = 1 << 30;
#pragma unroll
        for (int i = 0; i < R; ++i)
            if (v[i] > bv) {
                bv = v[i];
                be = lane + 32 * i;
            }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
            const int oe = __shfl_xor_sync(0xffffffffu, be, o);
            if (ov > bv || (ov == bv && oe < be)) {
                bv = ov;
                be = oe;
            }
        }
        if (be >= E) be = 0, bv = 0.0f;  // every logit is a NaN: any expert, weight zero
        put(k, be, bv / sum);
#pragma unroll
        for (int i = 0; i < R; ++i)
            if (lane + 32 * i == be) v[i] = -2.0f;
    }
}

// ---- prompt passes --------------------------------------------------------------------------------
template <int R>
__global__ void __launch_bounds__(128) moe_topk_kernel(const float *z, long ldz, int n, int E, int top, int *ids, float *weight, int *counts) {
    ptx::pdl_trigger();
    ptx::pdl_wait();
    const int t = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (t >= n) return;
    route_token<R>(z + static_cast<size_t>(t) * ldz, E, top, lane, [&](int k, int e, float w) {
        if (lane == 0) {
            ids[t * top + k] = e;
            weight[t * top + k] = w;
            atomicAdd(counts + e, 1);
        }
    });
}

// offs = exclusive sums of counts; cursor starts there; counts go back to zero for the next pass
__global__ void __launch_bounds__(1024) moe_scan_kernel(int *counts, int *offs, int *cursor, int E) {
    ptx::pdl_trigger();
    ptx::pdl_wait();
    __shared__ int s[kMaxExperts];
    const int e = threadIdx.x;
    int c = e < E ? counts[e] : 0;
    s[e] = c;
    __syncthreads();
    for (int o = 1; o < 1024; o <<= 1) {
        const int add = e >= o ? s[e - o] : 0;
        __syncthreads();
        s[e] += add;
        __syncthreads();
    }
    if (e < E) {
        offs[e] = cursor[e] = s[e] - c;
        counts[e] = 0;
        if (e == E - 1) offs[E] = s[e];
    }
}

// A block per token: its places in the sorted order, its row copied there (16-byte units).
__global__ void __launch_bounds__(128) moe_scatter_kernel(const int *ids, int top, int *cursor, int *place, int *token, const uint4 *x, long ldx16, int units,
                                                          uint4 *xs) {
    ptx::pdl_trigger();
    ptx::pdl_wait();
    __shared__ int s_place[kMaxTop];
    const int t = blockIdx.x;
    if (threadIdx.x < static_cast<unsigned>(top)) {
        const int p = atomicAdd(cursor + ids[t * top + threadIdx.x], 1);
        s_place[threadIdx.x] = p;
        place[t * top + threadIdx.x] = p;
        token[p] = t;
    }
    if (!xs) return;
    __syncthreads();
    for (int i = threadIdx.x; i < units; i += 128) {
        const uint4 v = x[static_cast<size_t>(t) * ldx16 + i];
        for (int k = 0; k < top; ++k) xs[static_cast<size_t>(s_place[k]) * units + i] = v;
    }
}

// ---- few tokens -------------------------------------------------------------------------------------
constexpr int kThreads = 512, kWarps = 16, kUnroll = 4;

struct FewMoeParams {
    const uint16_t *n;
    long ldn;
    int m;
    const float *z;
    long ldz;
    int experts, top;
    const uint16_t *up, *down, *sdown;
    size_t up_pitch, down_pitch, sdown_pitch;
    int up_chunks, down_chunks, sdown_chunks;
    int ff, width, ff_tiles, width_tiles;
    uint16_t *h;
    const uint16_t *hs;
    float *y;
    int *act;       // [0]: number of chosen experts, then (expert, 16 slots packed as bytes: 4 ints) each
};
constexpr int kActInts = 5;

// acc += W rows (r_lo, r_hi: this lane's two row pointers at its 8-column offset) x B rows, chunks of 32 columns
template <int NTL>
__device__ __forceinline__ void mma_chunk(float (&acc)[NTL][4], const uint4 &wl, const uint4 &wh, const uint4 (&b)[NTL]) {
    const uint32_t a0[4] = {wl.x, wh.x, wl.y, wh.y};
    const uint32_t a1[4] = {wl.z, wh.z, wl.w, wh.w};
#pragma unroll
    for (int j = 0; j < NTL; ++j) {
        ptx::mma_bf16(acc[j], a0, b[j].x, b[j].y);
        ptx::mma_bf16(acc[j], a1, b[j].z, b[j].w);
    }
}

template <int NTL, int R>
__global__ void __launch_bounds__(kThreads, 1) moe_few_up_kernel(const FewMoeParams p) {
    __shared__ float s_part[2][kWarps][NTL * 128];
    __shared__ int s_ids[LBK_GEMV_MAX_M][kMaxTop];
    __shared__ float s_wt[LBK_GEMV_MAX_M][kMaxTop];
    __shared__ unsigned s_mask[kMaxExperts];
    __shared__ short s_act[LBK_GEMV_MAX_M * kMaxTop];
    __shared__ int s_n;
    ptx::pdl_trigger();
    ptx::pdl_wait();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    for (int e = tid; e < p.experts; e += kThreads) s_mask[e] = 0u;
    __syncthreads();
    if (warp < p.m)
        route_token<R>(p.z + static_cast<size_t>(warp) * p.ldz, p.experts, p.top, lane, [&](int k, int e, float w) {
            if (lane == 0) {
                s_ids[warp][k] = e;
                s_wt[warp][k] = w;
                atomicOr(&s_mask[e], 1u << warp);
            }
        });
    __syncthreads();
    if (warp == 0) {  // the chosen experts in ascending order
        int cnt = 0;
        for (int e0 = 0; e0 < p.experts; e0 += 32) {
            const bool on = e0 + lane < p.experts && s_mask[e0 + lane] != 0u;
            const unsigned bal = __ballot_sync(0xffffffffu, on);
            if (on) s_act[cnt + __popc(bal & ((1u << lane) - 1u))] = static_cast<short>(e0 + lane);
            cnt += __popc(bal);
        }
        if (lane == 0) s_n = cnt;
    }
    __syncthreads();
    const int n_act = s_n;
    auto slot_of = [&](int tk, int e) {  // which of token tk's choices expert e is, -1: none
        if (tk >= p.m || !((s_mask[e] >> tk) & 1u)) return -1;
        int k = 0;
        while (k < p.top - 1 && s_ids[tk][k] != e) ++k;
        return k;
    };
    if (blockIdx.x == 0) {  // the list for the down kernel
        if (tid == 0) p.act[0] = n_act;
        for (int a = tid; a < n_act; a += kThreads) {
            const int e = s_act[a];
            p.act[1 + a * kActInts] = e;
            for (int w = 0; w < 4; ++w) {
                unsigned word = 0;
                for (int i = 0; i < 4; ++i) word |= (static_cast<unsigned>(slot_of(w * 4 + i, e)) & 255u) << (8 * i);
                p.act[2 + a * kActInts + w] = static_cast<int>(word);
            }
        }
    }
    const int c_per = (p.up_chunks + kWarps - 1) / kWarps;
    const int c0 = min(p.up_chunks, warp * c_per), c1 = min(p.up_chunks, c0 + c_per);
    int buf = 0;
    for (int unit = blockIdx.x; unit < n_act * p.ff_tiles; unit += gridDim.x, buf ^= 1) {
        const int a = unit / p.ff_tiles, tile = unit - a * p.ff_tiles, e = s_act[a];
        const unsigned mask = s_mask[e];
        float acc[NTL][4];
#pragma unroll
        for (int j = 0; j < NTL; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.0f;
        const size_t row0 = static_cast<size_t>(e) * p.ff;
        const uint16_t *wl_p = p.up + (row0 + min(tile * 16 + g, p.ff - 1)) * p.up_pitch + t * 8;
        const uint16_t *wh_p = p.up + (row0 + min(tile * 16 + g + 8, p.ff - 1)) * p.up_pitch + t * 8;
        for (int c = c0; c < c1; c += kUnroll) {
            uint4 wl[kUnroll], wh[kUnroll];
#pragma unroll
            for (int i = 0; i < kUnroll; ++i)
                if (c + i < c1) {
                    wl[i] = __ldcs(reinterpret_cast<const uint4 *>(wl_p + (c + i) * 32));
                    wh[i] = __ldcs(reinterpret_cast<const uint4 *>(wh_p + (c + i) * 32));
                }
#pragma unroll
            for (int i = 0; i < kUnroll; ++i)
                if (c + i < c1) {
                    uint4 b[NTL];
#pragma unroll
                    for (int j = 0; j < NTL; ++j) {
                        b[j] = make_uint4(0u, 0u, 0u, 0u);
                        if ((mask >> (j * 8 + g)) & 1u) b[j] = *reinterpret_cast<const uint4 *>(p.n + static_cast<size_t>(j * 8 + g) * p.ldn + (c + i) * 32 + t * 8);
                    }
                    mma_chunk<NTL>(acc, wl[i], wh[i], b);
                }
        }
        float *part = s_part[buf][warp];
#pragma unroll
        for (int j = 0; j < NTL; ++j) {
            part[j * 128 + (2 * t) * 16 + g] = acc[j][0];
            part[j * 128 + (2 * t + 1) * 16 + g] = acc[j][1];
            part[j * 128 + (2 * t) * 16 + g + 8] = acc[j][2];
            part[j * 128 + (2 * t + 1) * 16 + g + 8] = acc[j][3];
        }
        __syncthreads();
        for (int o = tid; o < NTL * 128; o += kThreads) {
            const int tk = o >> 4, r = tile * 16 + (o & 15);
            const int k = slot_of(tk, e);
            if (k < 0 || r >= p.ff) continue;
            float v = 0.0f;
#pragma unroll
            for (int w = 0; w < kWarps; ++w) v += s_part[buf][w][o];
            p.h[(static_cast<size_t>(tk) * p.top + k) * p.down_pitch + r] = dense::f32_bf16(dense::relu2(v) * s_wt[tk][k]);
        }
    }
}

template <int NTL>
__global__ void __launch_bounds__(kThreads, 1) moe_few_down_kernel(const FewMoeParams p) {
    __shared__ float s_part[2][kWarps][NTL * 128];
    __shared__ short s_e[LBK_GEMV_MAX_M * kMaxTop];
    __shared__ signed char s_slot[LBK_GEMV_MAX_M * kMaxTop][16];
    ptx::pdl_trigger();
    ptx::pdl_wait();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int n_act = p.act[0];
    for (int a = tid; a < n_act; a += kThreads) {
        s_e[a] = static_cast<short>(p.act[1 + a * kActInts]);
        for (int w = 0; w < 4; ++w) *reinterpret_cast<int *>(&s_slot[a][4 * w]) = p.act[2 + a * kActInts + w];
    }
    __syncthreads();
    const int cs = p.hs ? p.sdown_chunks : 0, ce = p.down_chunks, total = cs + n_act * ce;
    const int c_per = (total + kWarps - 1) / kWarps;
    const int c0 = min(total, warp * c_per), c1 = min(total, c0 + c_per);
    float gate[NTL][2];
#pragma unroll
    for (int j = 0; j < NTL; ++j)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int tk = j * 8 + 2 * t + i;
            gate[j][i] = p.hs && tk < p.m ? dense::sigmoid(p.z[static_cast<size_t>(tk) * p.ldz + p.experts]) : 0.0f;
        }
    int buf = 0;
    for (int tile = blockIdx.x; tile < p.width_tiles; tile += gridDim.x, buf ^= 1) {
        float acc[NTL][4], accs[NTL][4];
#pragma unroll
        for (int j = 0; j < NTL; ++j)
#pragma unroll
            for (int i = 0; i < 4; ++i) acc[j][i] = accs[j][i] = 0.0f;
        const int rl = min(tile * 16 + g, p.width - 1), rh = min(tile * 16 + g + 8, p.width - 1);
        for (int c = c0; c < c1; c += kUnroll) {
            uint4 wl[kUnroll], wh[kUnroll];
#pragma unroll
            for (int i = 0; i < kUnroll; ++i)
                if (c + i < c1) {
                    const uint16_t *a, *b;
                    if (c + i < cs) {
                        a = p.sdown + static_cast<size_t>(rl) * p.sdown_pitch + (c + i) * 32;
                        b = p.sdown + static_cast<size_t>(rh) * p.sdown_pitch + (c + i) * 32;
                    } else {
                        const int s = (c + i - cs) / ce, kk = c + i - cs - s * ce;
                        const size_t row0 = static_cast<size_t>(s_e[s]) * p.width;
                        a = p.down + (row0 + rl) * p.down_pitch + kk * 32;
                        b = p.down + (row0 + rh) * p.down_pitch + kk * 32;
                    }
                    wl[i] = __ldcs(reinterpret_cast<const uint4 *>(a + t * 8));
                    wh[i] = __ldcs(reinterpret_cast<const uint4 *>(b + t * 8));
                }
#pragma unroll
            for (int i = 0; i < kUnroll; ++i)
                if (c + i < c1) {
                    uint4 b[NTL];
                    if (c + i < cs) {
#pragma unroll
                        for (int j = 0; j < NTL; ++j) {
                            b[j] = make_uint4(0u, 0u, 0u, 0u);
                            if (j * 8 + g < p.m) b[j] = *reinterpret_cast<const uint4 *>(p.hs + static_cast<size_t>(j * 8 + g) * p.sdown_pitch + (c + i) * 32 + t * 8);
                        }
                        mma_chunk<NTL>(accs, wl[i], wh[i], b);
                    } else {
                        const int s = (c + i - cs) / ce, kk = c + i - cs - s * ce;
#pragma unroll
                        for (int j = 0; j < NTL; ++j) {
                            b[j] = make_uint4(0u, 0u, 0u, 0u);
                            const int k = s_slot[s][j * 8 + g];
                            if (k >= 0) b[j] = *reinterpret_cast<const uint4 *>(p.h + (static_cast<size_t>(j * 8 + g) * p.top + k) * p.down_pitch + kk * 32 + t * 8);
                        }
                        mma_chunk<NTL>(acc, wl[i], wh[i], b);
                    }
                }
        }
        float *part = s_part[buf][warp];
#pragma unroll
        for (int j = 0; j < NTL; ++j) {
            part[j * 128 + (2 * t) * 16 + g] = acc[j][0] + gate[j][0] * accs[j][0];
            part[j * 128 + (2 * t + 1) * 16 + g] = acc[j][1] + gate[j][1] * accs[j][1];
            part[j * 128 + (2 * t) * 16 + g + 8] = acc[j][2] + gate[j][0] * accs[j][2];
            part[j * 128 + (2 * t + 1) * 16 + g + 8] = acc[j][3] + gate[j][1] * accs[j][3];
        }
        __syncthreads();
        for (int o = tid; o < NTL * 128; o += kThreads) {
            const int tk = o >> 4, r = tile * 16 + (o & 15);
            if (tk >= p.m || r >= p.width) continue;
            float v = 0.0f;
#pragma unroll
            for (int w = 0; w < kWarps; ++w) v += s_part[buf][w][o];
            p.y[static_cast<size_t>(tk) * p.width + r] = v;
        }
    }
}

int check_route(size_t experts, size_t top) {
    if (experts == 0 || top == 0 || top > experts) return fail(LBK_ERR_INVALID, "routing %zu of %zu experts", top, experts);
    if (experts > static_cast<size_t>(kMaxExperts) || top > static_cast<size_t>(kMaxTop))
        return fail(LBK_ERR_UNSUPPORTED, "routing: at most %d experts, %d of them per token", kMaxExperts, kMaxTop);
    return LBK_OK;
}

}  // namespace

size_t moe_route_ints(size_t n, size_t experts, size_t top) { return 4 * n * top + 2 * (experts + 1) + kMaxExperts; }

// The counts come first and have room for every possible number of experts: they are zero at rest, whatever
// layer (with whatever number of experts) uses the block.
void moe_route_carve(MoeRoute &r, int *base, size_t n, size_t experts, size_t top) {
    r.counts = base;
    r.offs = r.counts + kMaxExperts;
    r.cursor = r.offs + experts + 1;
    r.ids = r.cursor + experts + 1;
    r.place = r.ids + n * top;
    r.token = r.place + n * top;
    r.weight = reinterpret_cast<float *>(r.token + n * top);
}

int launch_moe_route(Ctx *ctx, const float *z, long ldz, size_t n, size_t experts, size_t top, const MoeRoute &r, const void *x, long ldx, void *xs,
                     cudaStream_t st) {
    LBK_TRY(check_route(experts, top));
    if (n == 0) return LBK_OK;
    const dim3 grid(static_cast<unsigned>((n + 3) / 4));
    const int E = static_cast<int>(experts), k = static_cast<int>(top);
    if (E <= 256) LBK_CUDA(launch_chained(moe_topk_kernel<8>, grid, dim3(128), 0, st, z, ldz, static_cast<int>(n), E, k, r.ids, r.weight, r.counts));
    else LBK_CUDA(launch_chained(moe_topk_kernel<32>, grid, dim3(128), 0, st, z, ldz, static_cast<int>(n), E, k, r.ids, r.weight, r.counts));
    LBK_CUDA(launch_chained(moe_scan_kernel, dim3(1), dim3(1024), 0, st, r.counts, r.offs, r.cursor, E));
    LBK_CUDA(launch_chained(moe_scatter_kernel, dim3(static_cast<unsigned>(n)), dim3(128), 0, st, r.ids, k, r.cursor, r.place, r.token,
                            static_cast<const uint4 *>(x), ldx / 8, static_cast<int>(ldx / 8), static_cast<uint4 *>(xs)));
    LBK_CUDA(cudaGetLastError());
    ctx->launches += 3;
    return LBK_OK;
}

int launch_moe_few(Ctx *ctx, const MoeFewCall &c, cudaStream_t st) {
    LBK_TRY(check_route(static_cast<size_t>(c.experts), static_cast<size_t>(c.top)));
    if (c.m == 0) return LBK_OK;
    if (c.m > LBK_GEMV_MAX_M) return fail(LBK_ERR_INVALID, "the few-token expert kernels take up to %d tokens", LBK_GEMV_MAX_M);
    FewMoeParams p{};
    p.n = c.n;
    p.ldn = c.ldn;
    p.m = static_cast<int>(c.m);
    p.z = c.z;
    p.ldz = c.ldz;
    p.experts = c.experts;
    p.top = c.top;
    p.up = c.up.w;
    p.down = c.down.w;
    p.up_pitch = c.up.pitch;
    p.down_pitch = c.down.pitch;
    p.up_chunks = static_cast<int>(c.up.pitch / 32);
    p.down_chunks = static_cast<int>(c.down.pitch / 32);
    p.ff = static_cast<int>(c.ff);
    p.width = static_cast<int>(c.width);
    p.ff_tiles = (p.ff + 15) / 16;
    p.width_tiles = (p.width + 15) / 16;
    p.h = c.h;
    p.y = c.y;
    p.act = c.act;
    if (c.hs) {
        p.hs = c.hs;
        p.sdown = c.shared_down.w;
        p.sdown_pitch = c.shared_down.pitch;
        p.sdown_chunks = static_cast<int>(c.shared_down.pitch / 32);
    }
    const size_t most = c.m * c.top < static_cast<size_t>(c.experts) ? c.m * c.top : static_cast<size_t>(c.experts);
    const size_t units = most * p.ff_tiles;
    const dim3 gu(static_cast<unsigned>(units < static_cast<size_t>(ctx->sm_count) ? units : ctx->sm_count));
    const dim3 gd(static_cast<unsigned>(p.width_tiles < ctx->sm_count ? p.width_tiles : ctx->sm_count));
    const bool two = c.m > 8, wide = c.experts > 256;
    void (*up)(FewMoeParams) = two ? (wide ? moe_few_up_kernel<2, 32> : moe_few_up_kernel<2, 8>) : (wide ? moe_few_up_kernel<1, 32> : moe_few_up_kernel<1, 8>);
    LBK_CUDA(launch_chained(up, gu, dim3(kThreads), 0, st, p));
    LBK_CUDA(launch_chained(two ? moe_few_down_kernel<2> : moe_few_down_kernel<1>, gd, dim3(kThreads), 0, st, p));
    LBK_CUDA(cudaGetLastError());
    ctx->launches += 2;
    return LBK_OK;
}

size_t moe_few_act_ints(size_t m, size_t experts, size_t top) {
    const size_t most = m * top < experts ? m * top : experts;
    return 1 + most * kActInts;
}

}  // namespace lbk

using namespace lbk;

extern "C" size_t lbk_moe_route_ints(size_t n, size_t experts, size_t top) { return moe_route_ints(n, experts, top); }

extern "C" int lbk_moe_route(lbk_ctx *c, const float *z_dev, size_t z_pitch, size_t n, size_t experts, size_t top, int32_t *scratch_dev, const uint16_t *x_dev,
                             size_t x_pitch, uint16_t *sorted_dev, int32_t *ids_out_dev, float *weights_out_dev, int32_t *place_out_dev,
                             int32_t *offs_out_dev, void *stream) {
    if (!c) return fail(LBK_ERR_INVALID, "lbk_moe_route: context is null");
    if (n && (!z_dev || !scratch_dev || (sorted_dev && !x_dev))) return fail(LBK_ERR_INVALID, "lbk_moe_route: null buffer");
    if (sorted_dev && x_pitch % 64) return fail(LBK_ERR_SHAPE, "lbk_moe_route: rows of a multiple of 64 values");
    Ctx *ctx = reinterpret_cast<Ctx *>(c);
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    LBK_CUDA(cudaSetDevice(ctx->device));
    MoeRoute r;
    moe_route_carve(r, scratch_dev, n, experts, top);
    LBK_CUDA(cudaMemsetAsync(r.counts, 0, kMaxExperts * 4, st));
    LBK_TRY(launch_moe_route(ctx, z_dev, static_cast<long>(z_pitch), n, experts, top, r, x_dev, static_cast<long>(x_pitch), sorted_dev, st));
    if (ids_out_dev) LBK_CUDA(cudaMemcpyAsync(ids_out_dev, r.ids, n * top * 4, cudaMemcpyDeviceToDevice, st));
    if (weights_out_dev) LBK_CUDA(cudaMemcpyAsync(weights_out_dev, r.weight, n * top * 4, cudaMemcpyDeviceToDevice, st));
    if (place_out_dev) LBK_CUDA(cudaMemcpyAsync(place_out_dev, r.place, n * top * 4, cudaMemcpyDeviceToDevice, st));
    if (offs_out_dev) LBK_CUDA(cudaMemcpyAsync(offs_out_dev, r.offs, (experts + 1) * 4, cudaMemcpyDeviceToDevice, st));
    return LBK_OK;
}
