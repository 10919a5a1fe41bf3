// Projections with bf16 weights: y[t, r] = sum_k x[t, k] * W[r, k], f32 accumulation. Three kernels share one
// epilogue (lbk_dense_dev.cuh: f32 rows, activated rows in the compute type, or [q; k; v] rows of which k and v
// go straight into the cache):
//
//   dense_few_kernel   up to 8 tokens (decode, short portions). Bound: HBM, the weights once. 16 weight rows
//                      are the M side of mma.sync m16n8k16, the tokens its N side; a lane's 16-byte weight load
//                      is two MMAs' operands as it is (the contraction index may be permuted as long as both
//                      operands are permuted alike), so weights go global -> registers -> tensor core without
//                      shared memory or shuffles. The 16 warps of a CTA split K and meet in shared memory once per
//                      tile. Where whole tiles would leave SMs idle in the last round, the (tile, K) stream is cut into
//                      equal runs instead: a tile shared by several CTAs leaves partial sums in memory, and the one
//                      that arrives last adds them up in CTA order. The norms in front of the projection run in the prologue (at one or two tokens),
//                      while the CTA's first weight rows are on their way to L2.
//   dense_gemm_kernel  more tokens: tcgen05 (kind::f16), 128 weight rows x up to 256 tokens a tile, both operands
//                      by TMA (SWIZZLE_128B, 64 columns a stage), two accumulators in tensor memory so that the
//                      epilogue of one tile runs under the MMAs of the next, one persistent CTA per SM. A gated
//                      projection keeps gate and up accumulators of the same 128 rows side by side, so the
//                      product is taken where both sit in one thread's registers. Large calls are bound by the
//                      operands' way into the SMs (48 KB per 128 x 256 x 64 block): they take the wide form, two
//                      weight boxes x up to 256 tokens (64 KB for twice the block), whose accumulators fill tensor
//                      memory, so its epilogue is not hidden; choose_tile weighs the two. Few tiles and a long K (a short
//                      portion of a prompt) are cut along K over a cluster of 2 to 8 CTAs, whose accumulators meet
//                      in shared memory: every CTA reads its share of the tokens from all of them, in rank order.
//                      With experts the tokens
//                      arrive sorted and the tile list comes from the device-side counts.
//   dense_f32_kernel   everything in 32-bit (FMA), for LBK_COMPUTE_F32.
#include "lbk_dense.cuh"
#include "lbk_dense_dev.cuh"
#include "lbk_ptx.cuh"
#include "lbk_tcgen05.cuh"

namespace lbk {

namespace {

using namespace tc;

// ---- few tokens ---------------------------------------------------------------------------------
constexpr int kFewThreads = 512, kFewWarps = 16;
constexpr int kFewTokens = 8;               // up to here; 9 to 16 tokens run faster on dense_gemm_kernel (14336 -> 4096: 26 against 38 us)
constexpr int kFewPreMax = 2;               // tokens whose norms run in the prologue
constexpr size_t kFewXSmem = 96 * 1024;     // activations in shared memory up to this, else read through L1

constexpr int kFewPart = 2 * 128;           // floats of a partial tile: gate and up, 8 tokens, 16 rows
constexpr int kFewMaxTiles = 1 << 14, kFewMaxCtas = 512;
constexpr int kFewPrefetch = 2;             // 128-byte lines a thread asks L2 for ahead of the kernel in front

struct FewParams {
    const uint16_t *w;
    size_t pitch;
    int out_rows, up_row, chunks, tiles, m;
    const uint16_t *x;
    long ldx;
    int x_smem, xs_stride;                  // bytes per token row in shared memory
    int per;                                // 32-column chunks of the (tile, K) stream a CTA takes
    float *parts;                           // [2 * CTAs][kFewPart] partial sums of tiles shared between CTAs
    int *counters;                          // [tiles], zero at rest
    DenseEpi epi;
    DensePre pre;
    int n;                                  // columns of the normed row
};

// One token's row: the norms of DensePre, the result as bf16 into shared memory (and nout). 512 threads, up to
// four float4 each (rows of at most 8192 values).
__device__ __forceinline__ void few_norm_row(const FewParams &p, int t, bool writer, uint16_t *dst, float *s_red) {
    const int n4 = p.n >> 2, tid = threadIdx.x;
    const float inv_n = 1.0f / static_cast<float>(p.n);
    const float4 *xr = reinterpret_cast<const float4 *>(p.pre.x + static_cast<size_t>(t) * p.n);
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    float4 v[4], u[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const int i = tid + j * kFewThreads;
        u[j] = i < n4 ? xr[i] : zero;
    }
    if (p.pre.mode == kPreAddNorm) {
        const float4 *yr = reinterpret_cast<const float4 *>(p.pre.y + static_cast<size_t>(t) * p.n);
        float s = 0.0f;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int i = tid + j * kFewThreads;
            v[j] = i < n4 ? yr[i] : zero;
            s += (v[j].x + v[j].y) + (v[j].z + v[j].w);
        }
        const float mean = p.pre.rms ? 0.0f : dense::block_sum<kFewThreads>(s, s_red) * inv_n;
        float ss = 0.0f;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int i = tid + j * kFewThreads;
            v[j] = i < n4 ? make_float4(v[j].x - mean, v[j].y - mean, v[j].z - mean, v[j].w - mean) : zero;
            ss += (v[j].x * v[j].x + v[j].y * v[j].y) + (v[j].z * v[j].z + v[j].w * v[j].w);
        }
        const float r = 1.0f / sqrtf(dense::block_sum<kFewThreads>(ss, s_red) * inv_n + p.pre.eps);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int i = tid + j * kFewThreads;
            if (i < n4) {
                const float4 g = __ldg(reinterpret_cast<const float4 *>(p.pre.w_post) + i);
                u[j] = make_float4(u[j].x + v[j].x * r * g.x, u[j].y + v[j].y * r * g.y, u[j].z + v[j].z * r * g.z, u[j].w + v[j].w * r * g.w);
                if (writer) reinterpret_cast<float4 *>(p.pre.xout + static_cast<size_t>(t) * p.n)[i] = u[j];
            }
        }
    }
    float r = 1.0f;
    if (p.pre.w) {
        float mean = 0.0f;
        if (!p.pre.rms) {
            float s = 0.0f;
#pragma unroll
            for (int j = 0; j < 4; ++j) s += (u[j].x + u[j].y) + (u[j].z + u[j].w);
            mean = dense::block_sum<kFewThreads>(s, s_red) * inv_n;
        }
        float ss = 0.0f;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int i = tid + j * kFewThreads;
            u[j] = i < n4 ? make_float4(u[j].x - mean, u[j].y - mean, u[j].z - mean, u[j].w - mean) : zero;
            ss += (u[j].x * u[j].x + u[j].y * u[j].y) + (u[j].z * u[j].z + u[j].w * u[j].w);
        }
        r = 1.0f / sqrtf(dense::block_sum<kFewThreads>(ss, s_red) * inv_n + p.pre.eps);
    }
    const int pad4 = p.chunks * 8;          // chunks of 32 columns: zeros past the row
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const int i = tid + j * kFewThreads;
        uint2 o = make_uint2(0u, 0u);
        if (i < n4) {
            const float4 g = p.pre.w ? __ldg(reinterpret_cast<const float4 *>(p.pre.w) + i) : make_float4(1.f, 1.f, 1.f, 1.f);
            o = make_uint2(dense::bf16_pair(u[j].x * r * g.x, u[j].y * r * g.y), dense::bf16_pair(u[j].z * r * g.z, u[j].w * r * g.w));
            if (writer && p.pre.nout) reinterpret_cast<uint2 *>(static_cast<uint16_t *>(p.pre.nout) + static_cast<size_t>(t) * p.pre.ldn)[i] = o;
        }
        if (i < pad4) reinterpret_cast<uint2 *>(dst)[i] = o;
    }
}

template <bool DUAL>
__global__ void __launch_bounds__(kFewThreads, 1) dense_few_kernel(const __grid_constant__ FewParams p) {
    extern __shared__ __align__(16) uint8_t few_smem[];
    __shared__ float s_red[32];
    constexpr int NA = DUAL ? 2 : 1;
    constexpr int kPart = NA * 128;         // floats a warp contributes per tile
    float *s_part = reinterpret_cast<float *>(few_smem);               // [2][16 warps][kPart]
    uint8_t *s_x = few_smem + 2 * kFewWarps * kPart * sizeof(float);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    ptx::pdl_trigger();
    const int s_begin = static_cast<int>(blockIdx.x) * p.per, s_end = min(p.tiles * p.chunks, s_begin + p.per);
    // the weights are constants: the first of this CTA's rows start moving to L2 while the kernel in front finishes
    {
        int at = s_begin, left = kFewPrefetch * kFewThreads;
        while (at < s_end && left > 0) {
            const int tile = at / p.chunks, a = at - tile * p.chunks, b = min(p.chunks, a + s_end - at);
            const int l0 = a / 2, lines = (b + 1) / 2 - l0;  // 128-byte lines of a row (pitch is a multiple of 64 columns)
#pragma unroll
            for (int w = 0; w < NA; ++w)
                for (int i = tid; i < 16 * lines; i += kFewThreads) {
                    const int r = min(tile * 16 + i / lines, p.out_rows - 1) + w * p.up_row;
                    asm volatile("prefetch.global.L2 [%0];" ::"l"(p.w + static_cast<size_t>(r) * p.pitch + (l0 + i % lines) * 64));
                }
            left -= NA * 16 * lines;
            at += b - a;
        }
    }
    ptx::pdl_wait();
    int pos0;
    if (!dense::rows_fit(p.epi, p.m, pos0)) return;
    if (p.pre.mode != kPreNone) {
        for (int tk = 0; tk < p.m; ++tk) few_norm_row(p, tk, blockIdx.x == 0, reinterpret_cast<uint16_t *>(s_x + tk * p.xs_stride), s_red);
        __syncthreads();
    } else if (p.x_smem) {
        const int units = p.chunks * 4;     // 16-byte units per row
        for (int i = tid; i < p.m * units; i += kFewThreads) {
            const int tk = i / units, c = i - tk * units;
            *reinterpret_cast<uint4 *>(s_x + tk * p.xs_stride + c * 16) = *reinterpret_cast<const uint4 *>(p.x + static_cast<size_t>(tk) * p.ldx + c * 8);
        }
        __syncthreads();
    }
    __shared__ int s_last;
    // The CTA's run of the stream is a sequence of tile parts, a warp's share of one part a sequence of steps of U
    // chunks. The loads of a step are issued one step ahead, across tiles too: a warp always has two steps in flight.
    constexpr int U = DUAL ? 2 : 4;
    struct Step {
        int tile, k0, k1, c, c1;
    };
    int at = s_begin;
    auto next_part = [&](Step &q) {
        q.tile = at / p.chunks;
        q.k0 = at - q.tile * p.chunks;
        q.k1 = min(p.chunks, q.k0 + s_end - at);
        at += q.k1 - q.k0;
        const int c_per = (q.k1 - q.k0 + kFewWarps - 1) / kFewWarps;
        q.c = min(q.k1, q.k0 + warp * c_per);
        q.c1 = min(q.k1, q.c + c_per);
    };
    uint4 wl[NA][U], wh[NA][U], nl[NA][U], nh[NA][U];
    auto load = [&](const Step &q, uint4 (&lo)[NA][U], uint4 (&hi)[NA][U]) {
        const uint16_t *a = p.w + static_cast<size_t>(min(q.tile * 16 + g, p.out_rows - 1)) * p.pitch + t * 8;
        const uint16_t *b = p.w + static_cast<size_t>(min(q.tile * 16 + g + 8, p.out_rows - 1)) * p.pitch + t * 8;
        const size_t up = static_cast<size_t>(p.up_row) * p.pitch;
#pragma unroll
        for (int i = 0; i < U; ++i)
            if (q.c + i < q.c1) {
#pragma unroll
                for (int w = 0; w < NA; ++w) {
                    lo[w][i] = __ldcs(reinterpret_cast<const uint4 *>(a + w * up + (q.c + i) * 32));
                    hi[w][i] = __ldcs(reinterpret_cast<const uint4 *>(b + w * up + (q.c + i) * 32));
                }
            }
    };
    float acc[NA][4];
#pragma unroll
    for (int a = 0; a < NA; ++a)
        acc[a][0] = acc[a][1] = acc[a][2] = acc[a][3] = 0.0f;
    int buf = 0;
    Step cur, nxt;
    bool more = at < s_end;
    if (more) {
        next_part(cur);
        load(cur, wl, wh);
    }
    while (more) {
        nxt = cur;
        const bool part_done = cur.c + U >= cur.c1;
        if (!part_done) {
            nxt.c += U;
        } else if (at < s_end) {
            next_part(nxt);
        } else {
            more = false;
        }
        if (more) load(nxt, nl, nh);
#pragma unroll
        for (int i = 0; i < U; ++i)
            if (cur.c + i < cur.c1) {
                uint4 b = make_uint4(0u, 0u, 0u, 0u);
                if (g < p.m)
                    b = p.x_smem ? *reinterpret_cast<const uint4 *>(s_x + g * p.xs_stride + (cur.c + i) * 64 + t * 16)
                                 : *reinterpret_cast<const uint4 *>(p.x + static_cast<size_t>(g) * p.ldx + (cur.c + i) * 32 + t * 8);
#pragma unroll
                for (int a = 0; a < NA; ++a) {
                    const uint32_t a0[4] = {wl[a][i].x, wh[a][i].x, wl[a][i].y, wh[a][i].y};
                    const uint32_t a1[4] = {wl[a][i].z, wh[a][i].z, wl[a][i].w, wh[a][i].w};
                    ptx::mma_bf16(acc[a], a0, b.x, b.y);
                    ptx::mma_bf16(acc[a], a1, b.z, b.w);
                }
            }
        const int tile = cur.tile, k0 = cur.k0, k1 = cur.k1;
        cur = nxt;
#pragma unroll
        for (int w = 0; w < NA; ++w)
#pragma unroll
            for (int i = 0; i < U; ++i) {
                wl[w][i] = nl[w][i];
                wh[w][i] = nh[w][i];
            }
        if (!part_done) continue;
        // the sixteen K ranges meet: [warp][a][token][row], then one thread per output
        float *part = s_part + (buf * kFewWarps + warp) * kPart;
#pragma unroll
        for (int a = 0; a < NA; ++a) {
            float *o = part + a * 128;
            o[(2 * t) * 16 + g] = acc[a][0];
            o[(2 * t + 1) * 16 + g] = acc[a][1];
            o[(2 * t) * 16 + g + 8] = acc[a][2];
            o[(2 * t + 1) * 16 + g + 8] = acc[a][3];
            acc[a][0] = acc[a][1] = acc[a][2] = acc[a][3] = 0.0f;
        }
        buf ^= 1;         // the next part's sums go to the other buffer
        __syncthreads();  // ... whose readers passed this point one part ago
        const bool whole = k0 == 0 && k1 == p.chunks;
        static_assert(kFewTokens == 8, "one MMA tile of tokens; 128 (token, row) pairs, a thread each");
        const int o = tid, tk = o >> 4, r = tile * 16 + (o & 15);
        const bool mine = o < 128 && tk < p.m && r < p.out_rows;
        float v[NA];
        if (mine) {
#pragma unroll
            for (int a = 0; a < NA; ++a) {
                v[a] = 0.0f;
#pragma unroll
                for (int w = 0; w < kFewWarps; ++w) v[a] += s_part[((buf ^ 1) * kFewWarps + w) * kPart + a * 128 + o];
            }
        }
        if (!whole) {
            // a tile shared with neighbouring CTAs: a CTA's first tile has slot 2c, its last one slot 2c + 1
            auto slot = [&](int c) { return p.parts + static_cast<size_t>(2 * c + (c * p.per / p.chunks == tile ? 0 : 1)) * kFewPart; };
            float *own = slot(blockIdx.x);
            if (mine) {
#pragma unroll
                for (int a = 0; a < NA; ++a) __stcg(own + a * 128 + o, v[a]);
            }
            __threadfence();
            __syncthreads();
            const int first = tile * p.chunks / p.per, last = ((tile + 1) * p.chunks - 1) / p.per;
            if (tid == 0) {
                const int before = atomicAdd(p.counters + tile, 1);
                s_last = before == last - first;
                if (s_last) p.counters[tile] = 0;
            }
            __syncthreads();
            if (!s_last) continue;
            __threadfence();
            if (mine) {
#pragma unroll
                for (int a = 0; a < NA; ++a) v[a] = 0.0f;
                for (int c = first; c <= last; ++c) {
                    const float *q = slot(c);
#pragma unroll
                    for (int a = 0; a < NA; ++a) v[a] += __ldcg(q + a * 128 + o);
                }
            }
        }
        if (mine) {
            const float val = DUAL ? dense::gelu_tanh<false>(v[0]) * v[NA - 1] : v[0];
            dense::row_store<uint16_t>(p.epi, dense::row_plan<uint16_t>(p.epi, r, pos0), tk, val);
        }
    }
}

// ---- many tokens: tcgen05 -------------------------------------------------------------------------
constexpr int kGRows = 128;                     // weight rows per box (MMA M, TMEM lanes)
constexpr int kGWBytes = kGRows * 128;          // 16 KB: 128 rows x 64 columns
constexpr int kGRing = 192 * 1024;              // four stages of 48 KB (one weight box + 256 tokens, or two + 128), wide: three of 64 KB
constexpr int kGBars = kGRing;
constexpr int kGMisc = kGBars + 32 * 8;
constexpr int kGMaxExperts = 1024;
constexpr int kGSplitCtas = 128;                // CTAs of a launch that splits K over clusters
constexpr int kGSmem = kGMisc + 64 + 1024;
constexpr int kGEpiWarps = 8, kGTmaWarp = 8, kGMmaWarp = 9;
constexpr int kGThreads = 10 * 32;
constexpr int kGated = 1, kWide = 2;            // KIND bits

struct GemmParams {
    CUtensorMap w;      // bytes [stacked rows][pitch * 2], box [128][128]
    CUtensorMap x;      // bytes [tokens][ldx * 2], box [nt][128]
    DenseEpi epi;
    int out_rows, box2_row, tile_rows, k_blocks, m, nt, row_tiles, token_tiles, tiles;  // box2_row: rows from the first weight box to the second
    int experts, group_rows;
    const int *offs;
    int *err_word;
    int ksplit, kb_part;    // CTAs per tile (the cluster's size), K blocks each
};

__device__ __forceinline__ void cluster_sync() {
    asm volatile("barrier.cluster.arrive.release;\nbarrier.cluster.wait.acquire;" ::: "memory");
}
__device__ __forceinline__ uint32_t peer_smem(uint32_t addr, int rank) {
    uint32_t d;
    asm("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(d) : "r"(addr), "r"(rank));
    return d;
}
__device__ __forceinline__ float ld_peer(uint32_t addr) {
    float v;
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr) : "memory");
    return v;
}

__device__ __forceinline__ void umma4(uint32_t d_tmem, uint64_t adesc, uint64_t bdesc, uint32_t idesc, uint32_t accumulate_first) {
    asm volatile(
        "{\n"
        ".reg .pred p, q;\n"
        ".reg .b64 a1, a2, a3, b1, b2, b3;\n"
        "setp.ne.b32 p, %4, 0;\n"
        "setp.eq.b32 q, 0, 0;\n"
        "add.u64 a1, %1, 2;\n"
        "add.u64 a2, %1, 4;\n"
        "add.u64 a3, %1, 6;\n"
        "add.u64 b1, %2, 2;\n"
        "add.u64 b2, %2, 4;\n"
        "add.u64 b3, %2, 6;\n"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], a1, b1, %3, q;\n"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], a2, b2, %3, q;\n"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], a3, b3, %3, q;\n"
        "}\n" ::"r"(d_tmem), "l"(adesc), "l"(bdesc), "r"(idesc), "r"(accumulate_first)
        : "memory");
}

// A walk over this CTA's tiles that every role makes for itself: tile -> weight row, first token, tokens.
struct TileWalk {
    const GemmParams &p;
    const int *s_end;   // experts: running number of tiles
    int e = 0;
    __device__ TileWalk(const GemmParams &pp, const int *se) : p(pp), s_end(se) {}
    // tokens inside the tile: fastest, so that neighbouring CTAs share weight rows and tokens stay in L2
    __device__ __forceinline__ void get(int tile, int &row0, int &wrow, int &tok0, int &ntok) {
        if (!p.experts) {
            const int rt = tile / p.token_tiles, tt = tile - rt * p.token_tiles;
            row0 = wrow = rt * p.tile_rows;
            tok0 = tt * p.nt;
            ntok = min(p.nt, p.m - tok0);
            return;
        }
        while (tile >= s_end[e]) ++e;
        const int first = e ? s_end[e - 1] : 0, local = tile - first;
        const int b = p.offs[e], cnt = p.offs[e + 1] - b, tts = (cnt + p.nt - 1) / p.nt;
        const int rt = local / tts, tt = local - rt * tts;
        row0 = rt * p.tile_rows;
        wrow = e * p.group_rows + row0;
        tok0 = b + tt * p.nt;
        ntok = min(p.nt, cnt - tt * p.nt);
    }
};

template <int KIND, bool SPLIT>
__global__ void __launch_bounds__(kGThreads, 1) dense_gemm_kernel(const __grid_constant__ GemmParams p) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ int s_end[kGMaxExperts];
    constexpr bool GATED = (KIND & kGated) != 0, WIDE = (KIND & kWide) != 0;
    constexpr int NA = KIND ? 2 : 1;            // weight boxes a stage
    constexpr int kGStages = WIDE ? 3 : 4, kGStageBytes = kGRing / kGStages;
    constexpr int kXOff = NA * kGWBytes;
    constexpr int kAccCols = KIND == kGated ? 128 : 256;  // columns of one accumulator
    constexpr int NB = WIDE ? 1 : 2;            // sets of NA accumulators: NB * NA * kAccCols = 512 columns
    const uint32_t raw = ptx::smem_u32(smem_raw);
    const uint32_t base = (raw + 1023u) & ~1023u;
    uint8_t *sm = smem_raw + (base - raw);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const uint32_t bar0 = base + kGBars;
    volatile uint32_t *s_tmem = reinterpret_cast<volatile uint32_t *>(sm + kGMisc);
    volatile int *s_abort = reinterpret_cast<volatile int *>(sm + kGMisc + 4);
    auto bar = [&](int idx) { return bar0 + idx * 8; };
    constexpr int kFull = 0, kEmpty = kGStages, kAccFull = 2 * kGStages, kAccEmpty = 2 * kGStages + 2;
    if (tid == 0) {
        for (int i = 0; i < kGStages; ++i) {
            ptx::mbar_init(bar(kFull + i), 1);
            ptx::mbar_init(bar(kEmpty + i), 1);
        }
        for (int a = 0; a < 2; ++a) {
            ptx::mbar_init(bar(kAccFull + a), 1);
            ptx::mbar_init(bar(kAccEmpty + a), kGEpiWarps);
        }
        *s_abort = 0;
        ptx::fence_barrier_init();
    }
    if (warp == kGMmaWarp) {
        tmem_alloc(base + kGMisc, 512);
        tmem_relinquish();
    }
    int tiles = p.tiles;
    if (p.experts) {
        ptx::pdl_wait();  // the counts are the kernel's in front
        for (int e = tid; e < p.experts; e += kGThreads) s_end[e] = (p.offs[e + 1] - p.offs[e] + p.nt - 1) / p.nt * p.row_tiles;
        __syncthreads();
        if (tid == 0)
            for (int e = 1; e < p.experts; ++e) s_end[e] += s_end[e - 1];
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    if (p.experts) tiles = s_end[p.experts - 1];
    const uint32_t tmem_base = *s_tmem;
    ptx::pdl_trigger();
    bool ok = true;
    TileWalk walk(p, s_end);
    // this CTA's tiles and K blocks; SPLIT: one tile per cluster, a part of its K per CTA
    const int rank = SPLIT ? static_cast<int>(blockIdx.x) % p.ksplit : 0;
    const int first = SPLIT ? static_cast<int>(blockIdx.x) / p.ksplit : static_cast<int>(blockIdx.x);
    const int step = SPLIT ? tiles : static_cast<int>(gridDim.x);
    const int kb0 = SPLIT ? rank * p.kb_part : 0;
    const int kbn = SPLIT ? min(p.kb_part, p.k_blocks - kb0) : p.k_blocks;

    if (warp == kGTmaWarp) {
        // ================= TMA producer =================
        if (lane == 0) {
            const int my_tiles = tiles > first ? (tiles - first + step - 1) / step : 0;
            const int total = my_tiles * kbn;
            const uint32_t stage_tx = static_cast<uint32_t>(NA * kGWBytes + p.nt * 128);
            int row0, wrow = 0, tok0 = 0, ntok, s = 0, round = 0, kb = 0, tile = first;
            // Without experts the weights' first ring is on its way before the kernel in front is known to be complete.
            const int pre = p.experts ? 0 : (total < kGStages ? total : kGStages);
            for (int it = 0; it < pre; ++it) {
                walk.get(first + (it / kbn) * step, row0, wrow, tok0, ntok);
                ptx::mbar_arrive_expect_tx(bar(kFull + it), stage_tx);
#pragma unroll
                for (int a = 0; a < NA; ++a)
                    ptx::tma_load_2d(base + it * kGStageBytes + a * kGWBytes, &p.w, bar(kFull + it), (kb0 + it % kbn) * 128, wrow + a * p.box2_row);
            }
            if (!p.experts) ptx::pdl_wait();
            for (int it = 0; it < total; ++it) {
                if (kb == 0) walk.get(tile, row0, wrow, tok0, ntok);
                const uint32_t st = base + s * kGStageBytes;
                if (it >= pre) {
                    if (round > 0 && !wait_bar(bar(kEmpty + s), (round - 1) & 1, s_abort)) {
                        ok = false;
                        break;
                    }
                    ptx::mbar_arrive_expect_tx(bar(kFull + s), stage_tx);
#pragma unroll
                    for (int a = 0; a < NA; ++a) ptx::tma_load_2d(st + a * kGWBytes, &p.w, bar(kFull + s), (kb0 + kb) * 128, wrow + a * p.box2_row);
                }
                ptx::tma_load_2d(st + kXOff, &p.x, bar(kFull + s), (kb0 + kb) * 128, tok0);
                if (++s == kGStages) {
                    s = 0;
                    ++round;
                }
                if (++kb == kbn) {
                    kb = 0;
                    tile += step;
                }
            }
        }
    } else if (warp == kGMmaWarp) {
        // ================= MMA issuer (one thread) =================
        if (lane == 0) {
            const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | (static_cast<uint32_t>(p.nt >> 3) << 17) | ((kGRows >> 4) << 24);
            const uint64_t adesc0 = smem_desc_sw128(base), bdesc0 = smem_desc_sw128(base + kXOff);
            int s = 0, phase = 0, tcount = 0;
            for (int tile = first; tile < tiles && ok; tile += step, ++tcount) {
                const int a = tcount % NB, around = tcount / NB;
                if (around > 0 && !wait_bar(bar(kAccEmpty + a), (around - 1) & 1, s_abort)) {
                    ok = false;
                    break;
                }
                tc_fence_after();
                const uint32_t d_tmem = tmem_base + a * 256;
                for (int kb = 0; kb < kbn; ++kb) {
                    if (!wait_bar(bar(kFull + s), phase, s_abort)) {
                        ok = false;
                        break;
                    }
                    tc_fence_after();
                    const uint64_t off = static_cast<uint64_t>(s) * (kGStageBytes >> 4);
#pragma unroll
                    for (int w2 = 0; w2 < NA; ++w2)
                        umma4(d_tmem + w2 * kAccCols, adesc0 + off + static_cast<uint64_t>(w2 * (kGWBytes >> 4)), bdesc0 + off, idesc, kb ? 1u : 0u);
                    umma_commit(bar(kEmpty + s));
                    if (++s == kGStages) {
                        s = 0;
                        phase ^= 1;
                    }
                }
                if (!ok) break;
                umma_commit(bar(kAccFull + a));
            }
        }
    } else {
        // ================= epilogue (warps w and w + 4: TMEM lane quadrant w & 3) =================
        if (!p.experts) ptx::pdl_wait();  // outputs may still be read by the kernel in front; the position is its
        int pos0 = 0;
        const bool fits = dense::rows_fit(p.epi, p.m, pos0);
        const int quad = warp & 3, half = warp >> 2;  // half: one of two plain weight boxes, or every second 32 tokens
        int tcount = 0;
        for (int tile = first; tile < tiles && ok; tile += step, ++tcount) {
            const int a = tcount % NB, around = tcount / NB;
            int row0, wrow, tok0, ntok;
            walk.get(tile, row0, wrow, tok0, ntok);
            if (!__all_sync(0xffffffffu, wait_bar(bar(kAccFull + a), around & 1, s_abort))) {
                ok = false;
                break;
            }
            tc_fence_after();
            if (SPLIT) {
                // this part's sums to shared memory, [accumulator][token][row] (the ring is free: every MMA has retired)
                const uint32_t acc = tmem_base + (static_cast<uint32_t>(quad * 32) << 16);
                float *mine = reinterpret_cast<float *>(sm) + quad * 32 + lane;
#pragma unroll 1
                for (int w2 = 0; w2 < NA; ++w2)
#pragma unroll 1
                    for (int c = half; c * 32 < ntok; c += 2) {
                        uint32_t v[32];
                        tmem_ld32(acc + w2 * kAccCols + c * 32, v);
                        tmem_ld_wait();
#pragma unroll
                        for (int i = 0; i < 32; ++i)
                            if (c * 32 + i < p.nt) mine[(w2 * p.nt + c * 32 + i) * kGRows] = __uint_as_float(v[i]);
                    }
                tc_fence_before();
                break;
            }
            const int row = row0 + (KIND == kWide ? half * kGRows : 0) + quad * 32 + lane;
            dense::RowPlan plan;
            if (row < p.out_rows && fits) plan = dense::row_plan<uint16_t>(p.epi, row, pos0);
            const uint32_t acc = tmem_base + (static_cast<uint32_t>(quad * 32) << 16) + (KIND == kWide ? half * kAccCols : a * 256);
#pragma unroll 1
            for (int c = KIND == kWide ? 0 : half; c * 32 < ntok; c += KIND == kWide ? 1 : 2) {
                uint32_t v[32];
                tmem_ld32(acc + c * 32, v);
                if (GATED) {
                    uint32_t u[32];
                    tmem_ld32(acc + kAccCols + c * 32, u);
                    tmem_ld_wait();
#pragma unroll
                    for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(dense::gelu_tanh<false>(__uint_as_float(v[i])) * __uint_as_float(u[i]));
                } else {
                    tmem_ld_wait();
                }
                dense::row_store_run<uint16_t>(p.epi, plan, tok0 + c * 32, ntok - c * 32, v);
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) ptx::mbar_arrive(bar(kAccEmpty + a));
        }
    }
    if (SPLIT) {
        cluster_sync();  // every part's sums are in its CTA's shared memory
        if (warp < kGEpiWarps) {
            int pos0 = 0, row0, wrow, tok0, ntok;
            const bool fits = dense::rows_fit(p.epi, p.m, pos0);
            walk.get(first, row0, wrow, tok0, ntok);
            const int lane_row = (warp & 3) * 32 + lane, row = row0 + lane_row;
            const int per = (ntok + p.ksplit - 1) / p.ksplit, t0 = rank * per, t1 = min(ntok, t0 + per);  // this CTA's tokens
            if (row < p.out_rows && fits) {
                const dense::RowPlan plan = dense::row_plan<uint16_t>(p.epi, row, pos0);
                constexpr int TU = 4;  // tokens at a time: their loads from the other SMs are in flight together
                for (int t = t0 + (warp >> 2); t < t1; t += 2 * TU) {
                    float v[TU][NA];
#pragma unroll
                    for (int i = 0; i < TU; ++i)
#pragma unroll
                        for (int a = 0; a < NA; ++a) v[i][a] = 0.0f;
                    for (int r = 0; r < p.ksplit; ++r) {
                        const uint32_t peer = peer_smem(base + static_cast<uint32_t>(lane_row * 4), r);
                        float w[TU][NA];
#pragma unroll
                        for (int i = 0; i < TU; ++i)
#pragma unroll
                            for (int a = 0; a < NA; ++a)
                                w[i][a] = ld_peer(peer + static_cast<uint32_t>((a * p.nt + min(t + 2 * i, t1 - 1)) * kGRows * 4));
#pragma unroll
                        for (int i = 0; i < TU; ++i)
#pragma unroll
                            for (int a = 0; a < NA; ++a) v[i][a] += w[i][a];
                    }
#pragma unroll
                    for (int i = 0; i < TU; ++i)
                        if (t + 2 * i < t1)
                            dense::row_store<uint16_t>(p.epi, plan, tok0 + t + 2 * i, GATED ? dense::gelu_tanh<false>(v[i][0]) * v[i][NA - 1] : v[i][0]);
                }
            }
        }
        cluster_sync();  // nobody leaves while its sums are being read
    }
    if (!ok && lane == 0) atomicExch(p.err_word, 5);
    tc_fence_before();
    __syncthreads();
    if (warp == kGMmaWarp) {
        tc_fence_after();
        tmem_dealloc(tmem_base, 512);
    }
}

// ---- 32-bit ---------------------------------------------------------------------------------------
// 32 output rows x 32 tokens a block (256 threads, 2 x 2 values each), K in steps of 32 through shared memory.
struct F32Params {
    const uint16_t *w;
    size_t pitch;
    const float *x;
    long ldx;
    int cols, out_rows, up_row, m;
    DenseEpi epi;
    int experts, group_rows;
    const int *offs, *gather;
};
template <bool DUAL>
__global__ void __launch_bounds__(256) dense_f32_kernel(const F32Params p) {
    ptx::pdl_trigger();
    ptx::pdl_wait();
    constexpr int NA = DUAL ? 2 : 1;
    __shared__ float s_w[NA][32][33];
    __shared__ float s_x[32][33];
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int e = blockIdx.z;
    int first = 0, cnt = p.m;
    if (p.experts) {
        first = p.offs[e];
        cnt = p.offs[e + 1] - first;
    }
    const int r0 = blockIdx.x * 32, t0 = blockIdx.y * 32;
    if (t0 >= cnt) return;
    int pos0;
    if (!dense::rows_fit(p.epi, p.m, pos0)) return;
    const size_t wbase = static_cast<size_t>(e) * p.group_rows;
    float acc[NA][2][2] = {};
    for (int k0 = 0; k0 < p.cols; k0 += 32) {
        for (int i = tid; i < 1024; i += 256) {
            const int r = i >> 5, k = i & 31;
            const bool kin = k0 + k < p.cols;
#pragma unroll
            for (int a = 0; a < NA; ++a)
                s_w[a][r][k] = kin && r0 + r < p.out_rows ? dense::bf16_f32(p.w[(wbase + r0 + r + a * p.up_row) * p.pitch + k0 + k]) : 0.0f;
            float xv = 0.0f;
            if (kin && t0 + r < cnt) {
                const int sorted = first + t0 + r;
                xv = p.x[static_cast<size_t>(p.gather ? p.gather[sorted] : sorted) * p.ldx + k0 + k];
            }
            s_x[r][k] = xv;
        }
        __syncthreads();
#pragma unroll 8
        for (int k = 0; k < 32; ++k) {
            const float x0 = s_x[ty][k], x1 = s_x[ty + 16][k];
#pragma unroll
            for (int a = 0; a < NA; ++a) {
                const float w0 = s_w[a][tx][k], w1 = s_w[a][tx + 16][k];
                acc[a][0][0] = fmaf(w0, x0, acc[a][0][0]);
                acc[a][0][1] = fmaf(w0, x1, acc[a][0][1]);
                acc[a][1][0] = fmaf(w1, x0, acc[a][1][0]);
                acc[a][1][1] = fmaf(w1, x1, acc[a][1][1]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int r = r0 + tx + 16 * i;
        if (r >= p.out_rows) continue;
        const dense::RowPlan plan = dense::row_plan<float>(p.epi, r, pos0);
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const int t = t0 + ty + 16 * j;
            if (t >= cnt) continue;
            const float v = DUAL ? dense::gelu_tanh<true>(acc[0][i][j]) * acc[NA - 1][i][j] : acc[0][i][j];
            dense::row_store<float>(p.epi, plan, first + t, v);
        }
    }
}

int few_smem_bytes(const FewParams &p, bool dual) {
    return 2 * kFewWarps * (dual ? 2 : 1) * 128 * static_cast<int>(sizeof(float)) + (p.x_smem ? p.m * p.xs_stride : 0);
}

int launch_few(Ctx *ctx, const DenseCall &c, cudaStream_t st) {
    FewParams p{};
    p.w = c.w.w;
    p.pitch = c.w.pitch;
    p.out_rows = static_cast<int>(c.out_rows);
    p.up_row = static_cast<int>(c.up_row);
    p.chunks = static_cast<int>(c.w.pitch / 32);
    p.tiles = static_cast<int>((c.out_rows + 15) / 16);
    p.m = static_cast<int>(c.m);
    p.x = static_cast<const uint16_t *>(c.x);
    p.ldx = c.ldx;
    p.epi = c.epi;
    p.pre = c.pre;
    p.n = static_cast<int>(c.w.cols);
    p.xs_stride = static_cast<int>(c.w.pitch * 2 + 64);  // eight token rows start in different bank groups
    p.x_smem = c.pre.mode != kPreNone || c.m * p.xs_stride <= kFewXSmem;
    const size_t smem = static_cast<size_t>(few_smem_bytes(p, c.gated));
    // Whole tiles, or equal runs of the (tile, K) stream when the idle SMs of the last round would cost more than the
    // partial sums' trip through L2 (about 1.5 us; an SM streams about 40 bytes a nanosecond).
    int grid = ctx->sm_count;
    const int rounds = (p.tiles + grid - 1) / grid;
    const double tile_us = static_cast<double>(p.chunks) * 1024.0 * (c.gated ? 2 : 1) / 40e3;
    const double idle_us = (rounds - static_cast<double>(p.tiles) / grid) * tile_us;
    if (idle_us > 1.5 && p.tiles <= kFewMaxTiles && grid <= kFewMaxCtas && ctx->few_parts) {
        p.per = (p.tiles * p.chunks + grid - 1) / grid;
        p.parts = static_cast<float *>(ctx->few_parts);
        p.counters = reinterpret_cast<int *>(p.parts + static_cast<size_t>(2 * kFewMaxCtas) * kFewPart);
        grid = (p.tiles * p.chunks + p.per - 1) / p.per;
    } else {
        p.per = rounds * p.chunks;
        grid = (p.tiles + rounds - 1) / rounds;
    }
    void (*k)(FewParams) = c.gated ? dense_few_kernel<true> : dense_few_kernel<false>;
    LBK_CUDA(launch_chained(k, dim3(static_cast<unsigned>(grid)), dim3(kFewThreads), smem, st, p));
    LBK_CUDA(cudaGetLastError());
    ctx->launches++;
    return LBK_OK;
}

// CTAs a tile's K is cut over (a cluster), 1 when it is not worth it or the tiles are many: at most kGSplitCtas CTAs in
// all (clusters live inside a GPC, so not every SM can be part of one), at least four K blocks each.
int choose_ksplit(size_t tiles, int k_blocks, int boxes, int nt) {
    for (int s = 8; s >= 2; s >>= 1) {
        const int part = (k_blocks + s - 1) / s;
        if (tiles * s <= static_cast<size_t>(kGSplitCtas) && part >= 4 && part * (s - 1) < k_blocks && nt * boxes * kGRows * 4 <= kGRing) return s;
    }
    return 1;
}

// Tile shape: the one that finishes first, counting whole rounds of tiles over the SMs. Cycles per 64 columns of K: the
// MMAs' (two per token and weight box), or the operands' bytes at what an SM takes in beside 147 others (45 a cycle). The
// wide form adds its epilogue, a split K the exchange of the sums.
struct TileShape {
    int nt = 16, ksplit = 1;
    bool wide = false;
};
TileShape choose_tile(size_t m, size_t rows, int k_blocks, bool gated, int sms) {
    TileShape best;
    double best_cost = 1e30;
    for (int wide = 0; wide < 2; ++wide) {
        const int boxes = gated || wide ? 2 : 1, limit = boxes == 2 && !wide ? 128 : 256;
        const size_t tile_rows = wide && !gated ? 2 * kGRows : kGRows, row_tiles = (rows + tile_rows - 1) / tile_rows;
        for (int nt = 16; nt <= limit; nt += 16) {
            const size_t tiles = (m + nt - 1) / nt * row_tiles;
            const int ksplit = wide ? 1 : choose_ksplit(tiles, k_blocks, boxes, nt);
            const double mma = 2.0 * boxes * nt, bytes = (boxes * kGWBytes + nt * 128) / 45.0;
            double cost = static_cast<double>((tiles + sms - 1) / sms) * (mma > bytes ? mma : bytes) * k_blocks;
            if (ksplit > 1) cost = cost / ksplit + 3000.0 + 30.0 * boxes * nt;
            if (wide) cost += static_cast<double>((tiles + sms - 1) / sms) * (gated ? 7000.0 : 3000.0);
            if (cost <= best_cost) {
                best_cost = cost;
                best.nt = nt;
                best.ksplit = ksplit;
                best.wide = wide != 0;
            }
            if (static_cast<size_t>(nt) >= m) break;
        }
    }
    return best;
}

int launch_gemm_tc(Ctx *ctx, const DenseCall &c, cudaStream_t st) {
    if (c.experts > kGMaxExperts) return fail(LBK_ERR_UNSUPPORTED, "at most %d experts (got %d)", kGMaxExperts, c.experts);
    GemmParams p{};
    p.epi = c.epi;
    p.out_rows = static_cast<int>(c.out_rows);
    p.k_blocks = static_cast<int>(c.w.pitch / 64);
    p.m = static_cast<int>(c.m);
    p.ksplit = 1;
    p.kb_part = p.k_blocks;
    bool wide = false;
    const int limit = c.gated ? 128 : 256;
    if (c.experts) {
        // expected tokens per expert decide the tile; an expert with more takes several tiles
        const size_t each = (c.m + c.experts - 1) / c.experts;
        size_t nt = (each + each / 2 + 15) / 16 * 16;
        p.nt = static_cast<int>(nt < 32 ? 32 : nt > static_cast<size_t>(limit) ? limit : nt);
    } else {
        const TileShape t = choose_tile(c.m, c.out_rows, p.k_blocks, c.gated, ctx->sm_count);
        p.nt = t.nt;
        p.ksplit = t.ksplit;
        p.kb_part = (p.k_blocks + t.ksplit - 1) / t.ksplit;
        wide = t.wide;
    }
    p.tile_rows = wide && !c.gated ? 2 * kGRows : kGRows;
    p.box2_row = c.gated ? static_cast<int>(c.up_row) : kGRows;
    p.row_tiles = static_cast<int>((c.out_rows + p.tile_rows - 1) / p.tile_rows);
    p.token_tiles = static_cast<int>((c.m + p.nt - 1) / p.nt);
    p.tiles = p.row_tiles * p.token_tiles;
    p.experts = c.experts;
    p.group_rows = static_cast<int>(c.group_rows);
    p.offs = c.offs;
    p.err_word = ctx->err_word;
    LBK_TRY(encode_bytes_map(&p.w, c.w.w, c.w.pitch * 2, c.w.rows, c.w.pitch * 2, 128, kGRows));
    LBK_TRY(encode_bytes_map(&p.x, c.x, c.w.pitch * 2, c.m, static_cast<size_t>(c.ldx) * 2, 128, p.nt));
    if (p.ksplit > 1) {
        cudaLaunchConfig_t cfg{};
        cfg.gridDim = dim3(static_cast<unsigned>(p.tiles * p.ksplit));
        cfg.blockDim = dim3(kGThreads);
        cfg.dynamicSmemBytes = kGSmem;
        cfg.stream = st;
        cudaLaunchAttribute attr[2]{};
        attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[0].val.programmaticStreamSerializationAllowed = 1;
        attr[1].id = cudaLaunchAttributeClusterDimension;
        attr[1].val.clusterDim.x = static_cast<unsigned>(p.ksplit);
        attr[1].val.clusterDim.y = attr[1].val.clusterDim.z = 1;
        cfg.attrs = attr;
        cfg.numAttrs = 2;
        LBK_CUDA(cudaLaunchKernelEx(&cfg, c.gated ? dense_gemm_kernel<kGated, true> : dense_gemm_kernel<0, true>, p));
    } else {
        const int grid = !c.experts && p.tiles < ctx->sm_count ? p.tiles : ctx->sm_count;
        void (*k)(GemmParams) = wide ? (c.gated ? dense_gemm_kernel<kGated | kWide, false> : dense_gemm_kernel<kWide, false>)
                                     : (c.gated ? dense_gemm_kernel<kGated, false> : dense_gemm_kernel<0, false>);
        LBK_CUDA(launch_chained(k, dim3(static_cast<unsigned>(grid)), dim3(kGThreads),
                                static_cast<size_t>(kGSmem), st, p));
    }
    LBK_CUDA(cudaGetLastError());
    ctx->launches++;
    return LBK_OK;
}

int launch_f32(Ctx *ctx, const DenseCall &c, cudaStream_t st) {
    F32Params p{};
    p.w = c.w.w;
    p.pitch = c.w.pitch;
    p.x = static_cast<const float *>(c.x);
    p.ldx = c.ldx;
    p.cols = static_cast<int>(c.w.cols);
    p.out_rows = static_cast<int>(c.out_rows);
    p.up_row = static_cast<int>(c.up_row);
    p.m = static_cast<int>(c.m);
    p.epi = c.epi;
    p.experts = c.experts;
    p.group_rows = static_cast<int>(c.group_rows);
    p.offs = c.offs;
    p.gather = c.gather;
    // with experts an expert can have every token once (and no token twice)
    const dim3 grid(static_cast<unsigned>((c.out_rows + 31) / 32), static_cast<unsigned>((c.m + 31) / 32), static_cast<unsigned>(c.experts ? c.experts : 1));
    LBK_CUDA(launch_chained(c.gated ? dense_f32_kernel<true> : dense_f32_kernel<false>, grid, dim3(256), 0, st, p));
    LBK_CUDA(cudaGetLastError());
    ctx->launches++;
    return LBK_OK;
}

int dense_init(Ctx *ctx) {
    constexpr size_t parts = static_cast<size_t>(2 * kFewMaxCtas) * kFewPart * sizeof(float) + kFewMaxTiles * sizeof(int);
    LBK_CUDA(cudaMalloc(&ctx->few_parts, parts));
    LBK_CUDA(cudaMemset(ctx->few_parts, 0, parts));
    const int few_max = 2 * kFewWarps * 2 * 128 * 4 + static_cast<int>(kFewXSmem);
    LBK_CUDA(cudaFuncSetAttribute(dense_few_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, few_max));
    LBK_CUDA(cudaFuncSetAttribute(dense_few_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, few_max));
    if (static_cast<size_t>(kGSmem) > ctx->smem_optin) return fail(LBK_ERR_UNSUPPORTED, "dense GEMM kernel needs %d B of shared memory", kGSmem);
    for (void (*k)(GemmParams) : {dense_gemm_kernel<0, false>, dense_gemm_kernel<kGated, false>, dense_gemm_kernel<kWide, false>,
                                  dense_gemm_kernel<kGated | kWide, false>, dense_gemm_kernel<0, true>, dense_gemm_kernel<kGated, true>})
        LBK_CUDA(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, kGSmem));
    return LBK_OK;
}
const InitHook kInitDense(dense_init);

}  // namespace

bool dense_pre_supported(size_t m, size_t cols) { return m <= static_cast<size_t>(kFewPreMax) && cols % 4 == 0 && cols <= 8192; }

int launch_dense(Ctx *ctx, const DenseCall &c, cudaStream_t st) {
    if (c.m == 0 || c.out_rows == 0) return LBK_OK;
    if (!c.w.w || (!c.x && c.pre.mode == kPreNone)) return fail(LBK_ERR_INVALID, "dense projection: null buffer");
    if (c.compute == LBK_COMPUTE_F32) return launch_f32(ctx, c, st);
    if (c.pre.mode != kPreNone && (!dense_pre_supported(c.m, c.w.cols) || c.experts)) return fail(LBK_ERR_INVALID, "dense projection: this call cannot run the norms itself");
    if (c.m <= static_cast<size_t>(kFewTokens) && !c.experts) return launch_few(ctx, c, st);
    return launch_gemm_tc(ctx, c, st);
}

}  // namespace lbk

using namespace lbk;

extern "C" int lbk_dense_linear(lbk_ctx *c, int compute, const void *x_dev, size_t x_pitch, size_t m, const uint16_t *w_dev, size_t w_pitch,
                                size_t w_rows, size_t cols, int gated, size_t out_rows, int relu2, void *out_dev, size_t out_pitch, int out_f32,
                                const int32_t *expert_offs_dev, size_t experts, void *stream) {
    if (!c) return fail(LBK_ERR_INVALID, "lbk_dense_linear: context is null");
    Ctx *ctx = reinterpret_cast<Ctx *>(c);
    if (m && (!x_dev || !w_dev || !out_dev)) return fail(LBK_ERR_INVALID, "lbk_dense_linear: null buffer");
    if (w_pitch % 64 || w_pitch < cols || x_pitch < w_pitch || x_pitch % 64) return fail(LBK_ERR_SHAPE, "lbk_dense_linear: pitches are multiples of 64 columns that cover the row");
    if (experts && (gated || !expert_offs_dev || w_rows != experts * out_rows)) return fail(LBK_ERR_SHAPE, "lbk_dense_linear: stacked expert matrices of out_rows rows each");
    if (!experts && w_rows != out_rows * (gated ? 2 : 1)) return fail(LBK_ERR_SHAPE, "lbk_dense_linear: w has %zu rows for %zu outputs", w_rows, out_rows);
    LBK_CUDA(cudaSetDevice(ctx->device));
    DenseCall d;
    d.compute = compute;
    d.x = x_dev;
    d.ldx = static_cast<long>(x_pitch);
    d.m = m;
    d.w = DenseWeight{w_dev, w_rows, cols, w_pitch};
    d.gated = gated != 0;
    d.up_row = out_rows;
    d.out_rows = out_rows;
    d.epi.kind = out_f32 ? kEpiF32 : kEpiElem;
    d.epi.act = relu2 ? kActRelu2 : kActNone;
    d.epi.out = out_dev;
    d.epi.ld = static_cast<long>(out_pitch);
    d.experts = static_cast<int>(experts);
    d.group_rows = out_rows;
    d.offs = expert_offs_dev;
    return launch_dense(ctx, d, static_cast<cudaStream_t>(stream));
}

extern "C" int lbk_dense_linear_act(lbk_ctx *c, int compute, const void *x_dev, size_t x_pitch, size_t m, const uint16_t *w_dev, size_t w_pitch,
                                    size_t w_rows, size_t cols, const float *bias_dev, int act, size_t act_rows, void *out_dev, size_t out_pitch,
                                    int out_f32, void *stream) {
    if (!c) return fail(LBK_ERR_INVALID, "lbk_dense_linear_act: context is null");
    Ctx *ctx = reinterpret_cast<Ctx *>(c);
    if (m && (!x_dev || !w_dev || !out_dev)) return fail(LBK_ERR_INVALID, "lbk_dense_linear_act: null buffer");
    if (w_pitch % 64 || w_pitch < cols || x_pitch < w_pitch || x_pitch % 64) return fail(LBK_ERR_SHAPE, "lbk_dense_linear_act: pitches are multiples of 64 columns that cover the row");
    if (act != kActNone && act != kActRelu2 && act != kActSilu) return fail(LBK_ERR_INVALID, "lbk_dense_linear_act: unknown activation %d", act);
    LBK_CUDA(cudaSetDevice(ctx->device));
    DenseCall d;
    d.compute = compute;
    d.x = x_dev;
    d.ldx = static_cast<long>(x_pitch);
    d.m = m;
    d.w = DenseWeight{w_dev, w_rows, cols, w_pitch};
    d.out_rows = w_rows;
    d.epi.kind = out_f32 ? kEpiF32 : kEpiElem;
    d.epi.act = act;
    if (act_rows < w_rows) d.epi.act_rows = static_cast<int>(act_rows);
    d.epi.bias = bias_dev;
    d.epi.out = out_dev;
    d.epi.ld = static_cast<long>(out_pitch);
    return launch_dense(ctx, d, static_cast<cudaStream_t>(stream));
}
