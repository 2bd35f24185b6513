// Linear layers over bf16 weights on the sm_100a tensor cores (M > 8 rows, bf16 activations):
//     y[m, n] = sum_k x[m, k] W[n, k] (+ bias) (+ addend), f32 accumulation in TMEM;
// a GLU pair keeps gate and up columns of a tile side by side in one accumulator and applies the
// GLU in the epilogue, so neither projection is written to memory.
//
// Persistent: one CTA per SM walks the output tiles (128 rows x TN columns) of all layers of the
// group, rows fastest, so that consecutive CTAs share a weight tile in L2.
//   warp 0      TMA producer: 128B-swizzled boxes [128 x 64] of x and [TN x 64] of W per stage
//               (no multicast), completing on full[s].
//   warp 1      allocates TMEM, issues 4 tcgen05.mma (M=128, N=TN, K=16) per stage, commits the stage
//               to empty[s] and the tile to acc_full[b].
//   warps 2-5   epilogue of one accumulator while the other is being filled (2 x TN TMEM columns).
// Every wait is bounded like in mgq_gemm_tc.cu.
#include <cuda_fp16.h>

#include "mgq_linear.cuh"
#include "mgq_tcgen05.cuh"

namespace mgq {
namespace {

constexpr uint32_t TM = 128, TK = 64;
constexpr uint32_t kBytesA = TM * TK * 2;
constexpr int kThreads = 192;

__device__ unsigned int g_linear_tc_error = 0;

struct LinearMaps {
    CUtensorMap a[kMaxSegments], w[kMaxSegments];        // a GLU group has one layer: w[1] is its second weight
};

template <int TN> __host__ __device__ constexpr uint32_t stage_bytes() { return kBytesA + TN * TK * 2; }
template <int TN> __host__ __device__ constexpr int stages() { return TN == 256 ? 4 : TN == 128 ? 6 : 8; }

template <int S>
struct __align__(8) LinearShared {
    unsigned long long full[S], empty[S], acc_full[2], acc_empty[2];
    uint32_t tmem_base;
    volatile int failed;
};

constexpr uint32_t kStgBytes = 32 * 36 * 4;              // epilogue staging of one warp: 32 rows x 32 columns, padded rows

// Two values of a 2-byte output: bf16 for a GLU, f16 otherwise.
template <bool BF16> __device__ __forceinline__ uint32_t pack_pair(float x, float y)
{
    if (BF16) {
        const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
        return *reinterpret_cast<const uint32_t *>(&h);
    }
    const __half2 h = __floats2half2_rn(x, y);
    return *reinterpret_cast<const uint32_t *>(&h);
}

struct Tile {
    uint32_t si, m0, n0;
};

// Tile index -> layer, row block, column block (COLS output columns per tile).
template <uint32_t COLS>
__device__ __forceinline__ Tile find_tile(const LinearGroup &g, uint32_t tile, uint32_t mt)
{
    uint32_t nt = tile / mt, si = 0;
    const uint32_t m0 = (tile - nt * mt) * TM;
    while (si + 1 < g.count) {
        const uint32_t cols = (g.seg[si].n + COLS - 1) / COLS;
        if (nt < cols) break;
        nt -= cols;
        si++;
    }
    return Tile{si, m0, nt * COLS};
}

template <int TN, bool GLU>
__global__ void __launch_bounds__(kThreads, 1) linear_tc_kernel(const __grid_constant__ LinearMaps maps, const __grid_constant__ LinearGroup g,
                                                              uint32_t tiles)
{
    constexpr int S = stages<TN>();
    constexpr uint32_t COLS = GLU ? TN / 2 : TN, kStage = stage_bytes<TN>();
    extern __shared__ uint8_t smem_raw[];
    __shared__ LinearShared<S> sh;
    uint8_t *ring = reinterpret_cast<uint8_t *>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31u;

    if (tid == 0) {
        for (int s = 0; s < S; s++) {
            mbar_init(&sh.full[s], 1);
            mbar_init(&sh.empty[s], 1);
        }
        for (int b = 0; b < 2; b++) {
            mbar_init(&sh.acc_full[b], 1);
            mbar_init(&sh.acc_empty[b], 4);
        }
        sh.failed = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) tmem_alloc(&sh.tmem_base, 2 * TN);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = sh.tmem_base;
    pdl_launch_dependents();
    pdl_wait();
    uint32_t mt = (g.m + TM - 1) / TM;
    if (g.live) {                                        // fewer row blocks, so fewer tiles
        const uint32_t all = mt;
        mt = min(mt, (g.live[0] + g.live_add + TM - 1) / TM);
        tiles = tiles / all * mt;
    }

    if (warp == 0) {
        if (lane == 0) {
            uint32_t it = 0;
            int armed = -1;
            bool ok = true;
            for (uint32_t tile = blockIdx.x; tile < tiles && ok; tile += gridDim.x) {
                const Tile tl = find_tile<COLS>(g, tile, mt);
                const uint32_t nk = (g.seg[tl.si].k + TK - 1) / TK;
                for (uint32_t kc = 0; kc < nk; kc++, it++) {
                    const uint32_t s = it % S, ph = (it / S) & 1u;
                    ok = mbar_wait(&sh.empty[s], ph ^ 1u, &sh.failed, &g_linear_tc_error);
                    if (!ok) break;
                    uint8_t *st = ring + s * kStage;
                    mbar_arrive_expect_tx(&sh.full[s], kStage);
                    tma_load_2d(st, &maps.a[tl.si], (int)(kc * TK), (int)tl.m0, &sh.full[s]);
                    tma_load_2d(st + kBytesA, &maps.w[tl.si], (int)(kc * TK), (int)tl.n0, &sh.full[s]);
                    if (GLU) tma_load_2d(st + kBytesA + COLS * TK * 2, &maps.w[1], (int)(kc * TK), (int)tl.n0, &sh.full[s]);
                    armed = (int)it;
                }
            }
            // after a failure: let the copies in flight land before the CTA exits
            if (!ok)
                for (int i = armed; i >= 0 && i > armed - S; i--)
                    for (uint32_t w = 0; w < kWaitLimit && !mbar_try_wait(&sh.full[i % S], ((uint32_t)i / S) & 1u); w++) { }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            uint32_t it = 0, at = 0;
            bool ok = true;
            for (uint32_t tile = blockIdx.x; tile < tiles && ok; tile += gridDim.x, at++) {
                const uint32_t b = at & 1u;
                ok = mbar_wait(&sh.acc_empty[b], ((at >> 1) & 1u) ^ 1u, &sh.failed, &g_linear_tc_error);
                if (!ok) break;
                tc_fence_after();
                const uint32_t nk = (g.seg[find_tile<COLS>(g, tile, mt).si].k + TK - 1) / TK;
                for (uint32_t kc = 0; kc < nk; kc++, it++) {
                    const uint32_t s = it % S, ph = (it / S) & 1u;
                    ok = mbar_wait(&sh.full[s], ph, &sh.failed, &g_linear_tc_error);
                    if (!ok) break;
                    tc_fence_after();
                    const uint32_t base = smem_u32(ring + s * kStage);
#pragma unroll
                    for (uint32_t j = 0; j < TK / 16; j++)
                        umma_f16(tmem + b * TN, umma_desc(base + j * 32u), umma_desc(base + kBytesA + j * 32u), umma_instr(TM, TN),
                                 (kc | j) != 0 ? 1u : 0u);
                    umma_commit(&sh.empty[s]);
                }
                if (ok) umma_commit(&sh.acc_full[b]);
            }
        }
    } else {
        const uint32_t quad = warp & 3u;                 // TMEM lanes this warp may read
        float *stg = reinterpret_cast<float *>(ring + S * kStage) + quad * (kStgBytes / 4);
        uint32_t at = 0;
        for (uint32_t tile = blockIdx.x; tile < tiles; tile += gridDim.x, at++) {
            const uint32_t b = at & 1u;
            bool ok = mbar_wait(&sh.acc_full[b], (at >> 1) & 1u, &sh.failed, &g_linear_tc_error);
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) break;
            tc_fence_after();
            const Tile tl = find_tile<COLS>(g, tile, mt);
            const LinearSegment &sg = g.seg[tl.si];
            const uint32_t rbase = tl.m0 + quad * 32, n = sg.n;
            const uint32_t acc = tmem + ((quad * 32u) << 16) + b * TN;
            const bool narrow = (GLU && g.out_bf16) || (!GLU && g.out_f16);       // 2-byte outputs
#pragma unroll 1
            for (uint32_t c0 = 0; c0 < COLS; c0 += 32) {
                const uint32_t col = tl.n0 + c0;
                if (col >= n) break;                     // uniform over the warp
                const bool whole = col + 32 <= n && n % (narrow ? 8 : 4) == 0;
                // lane = row of the accumulator: bias and GLU here
                float y[32];
                tmem_ld32(acc + c0, y);
                if (GLU) {
                    float up[32];
                    tmem_ld32(acc + COLS + c0, up);
                    if (whole && sg.bias) {
#pragma unroll
                        for (int e = 0; e < 32; e += 4) {
                            const float4 bg = __ldg(reinterpret_cast<const float4 *>(sg.bias + col + e)), bu = __ldg(reinterpret_cast<const float4 *>(sg.bias2 + col + e));
                            y[e] += bg.x; y[e + 1] += bg.y; y[e + 2] += bg.z; y[e + 3] += bg.w;
                            up[e] += bu.x; up[e + 1] += bu.y; up[e + 2] += bu.z; up[e + 3] += bu.w;
                        }
                    } else if (sg.bias) {
#pragma unroll
                        for (int e = 0; e < 32; e++)
                            if (col + e < n) { y[e] += __ldg(sg.bias + col + e); up[e] += __ldg(sg.bias2 + col + e); }
                    }
#pragma unroll
                    for (int e = 0; e < 32; e++) y[e] = glu_f(y[e], up[e], g.act);
                } else if (sg.bias) {
                    if (whole) {
#pragma unroll
                        for (int e = 0; e < 32; e += 4) {
                            const float4 v = __ldg(reinterpret_cast<const float4 *>(sg.bias + col + e));
                            y[e] += v.x; y[e + 1] += v.y; y[e + 2] += v.z; y[e + 3] += v.w;
                        }
                    } else {
#pragma unroll
                        for (int e = 0; e < 32; e++)
                            if (col + e < n) y[e] += __ldg(sg.bias + col + e);
                    }
                }
                if (!GLU && g.out_f16) {
#pragma unroll
                    for (int e = 0; e < 32; e++) y[e] = fminf(fmaxf(y[e], -65504.f), 65504.f);
                }
                // through shared memory, so that a store instruction covers whole pieces of few rows
                if (whole && narrow) {
                    uint32_t *mine = reinterpret_cast<uint32_t *>(stg) + lane * 20;
#pragma unroll
                    for (int e = 0; e < 16; e += 4)
                        *reinterpret_cast<uint4 *>(mine + e) = make_uint4(pack_pair<GLU>(y[2 * e], y[2 * e + 1]), pack_pair<GLU>(y[2 * e + 2], y[2 * e + 3]),
                                                                          pack_pair<GLU>(y[2 * e + 4], y[2 * e + 5]), pack_pair<GLU>(y[2 * e + 6], y[2 * e + 7]));
                    __syncwarp();
#pragma unroll
                    for (int i = 0; i < 4; i++) {
                        const uint32_t r = i * 8 + lane / 4, piece = lane & 3u;
                        const uint4 v = *reinterpret_cast<const uint4 *>(reinterpret_cast<const uint32_t *>(stg) + r * 20 + piece * 4);
                        if (rbase + r < g.m) *reinterpret_cast<uint4 *>(static_cast<uint16_t *>(sg.out) + (size_t)(rbase + r) * n + col + piece * 8) = v;
                    }
                    __syncwarp();
                } else if (whole) {
                    float *mine = stg + lane * 36;
                    float4 add[8];
#pragma unroll
                    for (int i = 0; i < 8; i++) {        // all addends requested before the first one is needed
                        const uint32_t r = i * 4 + lane / 8;
                        add[i] = make_float4(0.f, 0.f, 0.f, 0.f);
                        if (!GLU && sg.addend && rbase + r < g.m) add[i] = *reinterpret_cast<const float4 *>(sg.addend + (size_t)(rbase + r) * n + col + (lane & 7u) * 4);
                    }
#pragma unroll
                    for (int e = 0; e < 32; e += 4) *reinterpret_cast<float4 *>(mine + e) = make_float4(y[e], y[e + 1], y[e + 2], y[e + 3]);
                    __syncwarp();
#pragma unroll
                    for (int i = 0; i < 8; i++) {
                        const uint32_t r = i * 4 + lane / 8;
                        float4 v = *reinterpret_cast<const float4 *>(stg + r * 36 + (lane & 7u) * 4);
                        v.x += add[i].x; v.y += add[i].y; v.z += add[i].z; v.w += add[i].w;
                        if (rbase + r < g.m) *reinterpret_cast<float4 *>(static_cast<float *>(sg.out) + (size_t)(rbase + r) * n + col + (lane & 7u) * 4) = v;
                    }
                    __syncwarp();
                } else if (rbase + lane < g.m) {         // ragged columns
                    const size_t o = (size_t)(rbase + lane) * n + col;
#pragma unroll
                    for (int e = 0; e < 32; e++) {
                        if (col + e >= n) continue;
                        if (narrow) static_cast<uint16_t *>(sg.out)[o + e] = (uint16_t)pack_pair<GLU>(y[e], 0.f);
                        else        static_cast<float *>(sg.out)[o + e] = !GLU && sg.addend ? y[e] + sg.addend[o + e] : y[e];
                    }
                }
            }
            tc_fence_before();
            if (lane == 0) mbar_arrive(&sh.acc_empty[b]);
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        __syncwarp();
        tc_fence_after();
        tmem_free(tmem, 2 * TN);
    }
}

int encode_rows(EncodeTiledFn encode, CUtensorMap &map, const void *base, uint32_t k, uint32_t ld, uint32_t rows, uint32_t box_rows)
{
    const cuuint64_t dims[2] = {k, rows};
    const cuuint64_t strides[1] = {(cuuint64_t)ld * 2};
    const cuuint32_t box[2] = {TK, box_rows};
    const cuuint32_t elem[2] = {1, 1};
    const CUresult cr = encode(&map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void *>(base), dims, strides, box, elem,
                               CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                               CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    return cr == CUDA_SUCCESS ? MGQ_OK : fail(MGQ_ERR_CUDA, "cuTensorMapEncodeTiled failed (%d)", (int)cr);
}

template <int TN, bool GLU>
int launch_tc(const LinearGroup &g, cudaStream_t stream)
{
    constexpr uint32_t COLS = GLU ? TN / 2 : TN;
    EncodeTiledFn encode = nullptr;
    if (int rc = encode_fn(encode)) return rc;
    LinearMaps maps{};
    uint32_t tiles = 0;
    for (uint32_t i = 0; i < g.count; i++) {
        const LinearSegment &s = g.seg[i];
        if (int rc = encode_rows(encode, maps.a[i], s.a, s.k, g.lda ? g.lda : s.k, g.m, TM)) return rc;
        if (int rc = encode_rows(encode, maps.w[i], s.w, s.k, s.k, s.n, COLS)) return rc;
        if (GLU)
            if (int rc = encode_rows(encode, maps.w[1], s.w2, s.k, s.k, s.n, COLS)) return rc;
        tiles += (s.n + COLS - 1) / COLS;
    }
    tiles *= (g.m + TM - 1) / TM;
    const size_t smem = (size_t)stages<TN>() * stage_bytes<TN>() + 4 * kStgBytes + 1024;
    if (int rc = allow_smem(linear_tc_kernel<TN, GLU>, smem)) return rc;
    return launch(linear_tc_kernel<TN, GLU>, dim3(min(tiles, 148u)), dim3(kThreads), smem, stream, maps, g, tiles);
}

template <bool GLU>
int launch_tc_sized(const LinearGroup &g, cudaStream_t stream)
{
    auto tiles = [&](uint32_t cols) {
        uint32_t t = 0;
        for (uint32_t i = 0; i < g.count; i++) t += (g.seg[i].n + cols - 1) / cols;
        return t * ((g.m + TM - 1) / TM);
    };
    const uint32_t f = GLU ? 2 : 1;
    if (tiles(256 / f) >= 148) return launch_tc<256, GLU>(g, stream);
    if (tiles(128 / f) >= 100) return launch_tc<128, GLU>(g, stream);
    return launch_tc<64, GLU>(g, stream);
}

}  // namespace

int launch_linear_tc(const LinearGroup &g, void *stream)
{
    for (uint32_t i = 0; i < g.count; i++)
        if (reinterpret_cast<uintptr_t>(g.seg[i].out) % 16 != 0 || reinterpret_cast<uintptr_t>(g.seg[i].addend) % 16 != 0)
            return fail(MGQ_ERR_ALIGN, "linear: outputs and addends must be 16-byte aligned");
    return g.glu ? launch_tc_sized<true>(g, static_cast<cudaStream_t>(stream)) : launch_tc_sized<false>(g, static_cast<cudaStream_t>(stream));
}

int linear_tc_status()
{
    unsigned int err = 0;
    MGQ_CUDA(cudaMemcpyFromSymbol(&err, g_linear_tc_error, sizeof err));
    if (!err) return MGQ_OK;
    const unsigned int zero = 0;
    MGQ_CUDA(cudaMemcpyToSymbol(g_linear_tc_error, &zero, sizeof zero));
    return fail(MGQ_ERR_TIMEOUT, "a bounded wait inside the tensor-core linear kernel ran out");
}

}  // namespace mgq
