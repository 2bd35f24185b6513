// Linear layers over bf16 weights stored [N, K]:  y[m, n] = sum_k x[m, k] W[n, k] (+ bias[n]) (+ addend[m, n]).
//
// One launch takes a GROUP of up to kMaxSegments independent layers that share M (the projections of
// one mixer: same or different inputs, different widths), so a decode step pays one kernel boundary
// for all of them.  A gated feed-forward's pair of projections runs as one segment with two weights
// whose epilogue applies the GLU.
//
//   linear_gemv_kernel   M <= 8: HBM-bound, a warp streams R weight rows with 16-byte loads for all M
//                        activation rows at once (every weight byte is read once per 8 rows).
//   linear_tiled_kernel  general: 64x64 register tiles in true f32 (f32 activations, sizes the tensor
//                        cores cannot take).
//   mgq_linear_tc.cu     M > 8, bf16 activations: tcgen05.
#include "mgq_linear.cuh"

namespace mgq {
namespace {

// ---------------------------------------------------------------- GEMV
// Unit = R weight rows of one segment (GLU: R/2 columns, gate and up rows of each).
template <typename XT, int M, int R, bool GLU, bool VEC>
__global__ void __launch_bounds__(128) linear_gemv_kernel(const __grid_constant__ LinearGroup g, uint32_t m, uint32_t row0)
{
    constexpr int COLS = GLU ? R / 2 : R;
    const uint32_t lane = threadIdx.x & 31u;
    uint32_t unit = blockIdx.x * 4u + (threadIdx.x >> 5), si = 0;
    pdl_launch_dependents();
    while (si < g.count) {
        const uint32_t units = (g.seg[si].n + COLS - 1) / COLS;
        if (unit < units) break;
        unit -= units;
        si++;
    }
    if (si >= g.count) return;
    const LinearSegment &s = g.seg[si];
    const uint32_t n0 = unit * COLS, k = s.k;
    const __nv_bfloat16 *w[R];
#pragma unroll
    for (int r = 0; r < R; r++) {
        const uint32_t n = min(n0 + (uint32_t)(GLU ? r / 2 : r), s.n - 1u);
        w[r] = static_cast<const __nv_bfloat16 *>((GLU && (r & 1)) ? s.w2 : s.w) + (size_t)n * k;
    }
    // weights are immutable: start moving the first pieces towards L2 before waiting for the activations
    if (lane * 64u < k) {
#pragma unroll
        for (int r = 0; r < R; r++) asm volatile("prefetch.global.L2 [%0];" ::"l"(w[r] + lane * 64u));
    }
    pdl_wait();
    const XT *x = static_cast<const XT *>(s.a) + (size_t)row0 * k;
    float acc[M][R];
#pragma unroll
    for (int i = 0; i < M; i++)
#pragma unroll
        for (int r = 0; r < R; r++) acc[i][r] = 0.f;
    if (VEC) {
        const uint32_t chunks = k / 8;
#pragma unroll(M <= 2 ? 4 : 2)
        for (uint32_t c = lane; c < chunks; c += 32) {
            uint4 q[R];
#pragma unroll
            for (int r = 0; r < R; r++)
                asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];"
                             : "=r"(q[r].x), "=r"(q[r].y), "=r"(q[r].z), "=r"(q[r].w) : "l"(w[r] + (size_t)c * 8));
#pragma unroll
            for (int i = 0; i < M; i++) {
                float xv[8];
                load8(x + (size_t)(i < (int)m ? i : 0) * k + (size_t)c * 8, xv);
#pragma unroll
                for (int r = 0; r < R; r++) {
                    float wv[8];
                    unpack8(q[r], wv);
#pragma unroll
                    for (int j = 0; j < 8; j++) acc[i][r] = fmaf(xv[j], wv[j], acc[i][r]);
                }
            }
        }
    } else {
        for (uint32_t c = lane; c < k; c += 32) {
            float wv[R];
#pragma unroll
            for (int r = 0; r < R; r++) wv[r] = __bfloat162float(w[r][c]);
#pragma unroll
            for (int i = 0; i < M; i++) {
                const float xv = to_f32(x[(size_t)(i < (int)m ? i : 0) * k + c]);
#pragma unroll
                for (int r = 0; r < R; r++) acc[i][r] = fmaf(xv, wv[r], acc[i][r]);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < M; i++)
#pragma unroll
        for (int r = 0; r < R; r++) acc[i][r] = warp_sum(acc[i][r]);
#pragma unroll
    for (int i = 0; i < M; i++) {
        if (i >= (int)m) break;
#pragma unroll
        for (int c = 0; c < COLS; c++) {
            const uint32_t n = n0 + c;
            if (lane != (uint32_t)(i * COLS + c) % 32u || n >= s.n) continue;
            const size_t o = (size_t)(row0 + i) * s.n + n;
            if (GLU) {
                const float y = glu_f(acc[i][2 * c] + (s.bias ? s.bias[n] : 0.f), acc[i][2 * c + 1] + (s.bias ? s.bias2[n] : 0.f), g.act);
                if (g.out_bf16) static_cast<__nv_bfloat16 *>(s.out)[o] = __float2bfloat16_rn(y);
                else            static_cast<float *>(s.out)[o] = y;
            } else {
                float y = acc[i][c];
                if (s.bias) y += s.bias[n];
                if (s.addend) y += s.addend[o];
                static_cast<float *>(s.out)[o] = y;
            }
        }
    }
}

template <typename XT, int M, int R, bool GLU>
int launch_gemv_vec(const LinearGroup &g, uint32_t m, uint32_t row0, bool vec, cudaStream_t stream)
{
    constexpr uint32_t COLS = GLU ? R / 2 : R;
    uint32_t units = 0;
    for (uint32_t i = 0; i < g.count; i++) units += (g.seg[i].n + COLS - 1) / COLS;
    const dim3 grid((units + 3) / 4);
    if (vec) return launch(linear_gemv_kernel<XT, M, R, GLU, true>, grid, dim3(128), 0, stream, g, m, row0);
    return launch(linear_gemv_kernel<XT, M, R, GLU, false>, grid, dim3(128), 0, stream, g, m, row0);
}

template <typename XT, int M>
int launch_gemv_rows(const LinearGroup &g, uint32_t m, uint32_t row0, bool vec, cudaStream_t stream)
{
    // enough warps to fill the GPU before a warp takes several rows
    uint32_t rows = 0;
    for (uint32_t i = 0; i < g.count; i++) rows += g.seg[i].n * (g.glu ? 2u : 1u);
    if (g.glu) {
        if (rows >= 9472u) return launch_gemv_vec<XT, M, 4, true>(g, m, row0, vec, stream);
        return launch_gemv_vec<XT, M, 2, true>(g, m, row0, vec, stream);
    }
    if (rows >= 9472u) return launch_gemv_vec<XT, M, 4, false>(g, m, row0, vec, stream);
    if (rows >= 4736u) return launch_gemv_vec<XT, M, 2, false>(g, m, row0, vec, stream);
    return launch_gemv_vec<XT, M, 1, false>(g, m, row0, vec, stream);
}

template <typename XT>
int launch_gemv_typed(const LinearGroup &g, bool vec, cudaStream_t stream)
{
    for (uint32_t row0 = 0; row0 < g.m; row0 += 8) {
        const uint32_t m = min(8u, g.m - row0);
        int rc;
        if (m == 1)      rc = launch_gemv_rows<XT, 1>(g, m, row0, vec, stream);
        else if (m == 2) rc = launch_gemv_rows<XT, 2>(g, m, row0, vec, stream);
        else if (m <= 4) rc = launch_gemv_rows<XT, 4>(g, m, row0, vec, stream);
        else             rc = launch_gemv_rows<XT, 8>(g, m, row0, vec, stream);
        if (rc) return rc;
    }
    return MGQ_OK;
}

// ---------------------------------------------------------------- general tiled kernel (CUDA cores, f32)
constexpr int BM = 64, BN = 64, BK = 16;

template <typename XT, bool GLU>
__global__ void __launch_bounds__(256) linear_tiled_kernel(const __grid_constant__ LinearGroup g)
{
    __shared__ float s_a[BK][BM + 4], s_w[GLU ? 2 : 1][BK][BN + 4];
    uint32_t tile = blockIdx.x, si = 0;
    pdl_launch_dependents();
    while (si < g.count) {
        const uint32_t tiles = (g.seg[si].n + BN - 1) / BN;
        if (tile < tiles) break;
        tile -= tiles;
        si++;
    }
    if (si >= g.count) return;
    const LinearSegment &s = g.seg[si];
    const uint32_t n0 = tile * BN, m0 = blockIdx.y * BM, k = s.k, t = threadIdx.x;
    const uint32_t tx = t & 15u, ty = t >> 4;
    const XT *a = static_cast<const XT *>(s.a);
    const __nv_bfloat16 *w = static_cast<const __nv_bfloat16 *>(s.w), *w2 = static_cast<const __nv_bfloat16 *>(s.w2);
    float acc[GLU ? 2 : 1][4][4];
#pragma unroll
    for (int u = 0; u < (GLU ? 2 : 1); u++)
#pragma unroll
        for (int i = 0; i < 4; i++)
#pragma unroll
            for (int j = 0; j < 4; j++) acc[u][i][j] = 0.f;
    pdl_wait();
    for (uint32_t k0 = 0; k0 < k; k0 += BK) {
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const uint32_t e = t + 256u * i, row = e / BK, kk = e % BK;
            const bool in_k = k0 + kk < k;
            s_a[kk][row] = in_k && m0 + row < g.m ? to_f32(a[(size_t)(m0 + row) * k + k0 + kk]) : 0.f;
            const bool in_w = in_k && n0 + row < s.n;
            s_w[0][kk][row] = in_w ? __bfloat162float(w[(size_t)(n0 + row) * k + k0 + kk]) : 0.f;
            if (GLU) s_w[GLU ? 1 : 0][kk][row] = in_w ? __bfloat162float(w2[(size_t)(n0 + row) * k + k0 + kk]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < BK; kk++) {
            const float4 av = *reinterpret_cast<const float4 *>(&s_a[kk][ty * 4]);
            const float ar[4] = {av.x, av.y, av.z, av.w};
#pragma unroll
            for (int u = 0; u < (GLU ? 2 : 1); u++) {
                const float4 wv = *reinterpret_cast<const float4 *>(&s_w[u][kk][tx * 4]);
                const float wr[4] = {wv.x, wv.y, wv.z, wv.w};
#pragma unroll
                for (int i = 0; i < 4; i++)
#pragma unroll
                    for (int j = 0; j < 4; j++) acc[u][i][j] = fmaf(ar[i], wr[j], acc[u][i][j]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const uint32_t row = m0 + ty * 4 + i;
        if (row >= g.m) break;
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const uint32_t n = n0 + tx * 4 + j;
            if (n >= s.n) break;
            const size_t o = (size_t)row * s.n + n;
            float y = acc[0][i][j];
            if (GLU) {
                y = glu_f(y + (s.bias ? s.bias[n] : 0.f), acc[GLU ? 1 : 0][i][j] + (s.bias ? s.bias2[n] : 0.f), g.act);
                if (g.out_bf16) static_cast<__nv_bfloat16 *>(s.out)[o] = __float2bfloat16_rn(y);
                else            static_cast<float *>(s.out)[o] = y;
                continue;
            }
            if (s.bias) y += s.bias[n];
            if (s.addend) y += s.addend[o];
            static_cast<float *>(s.out)[o] = y;
        }
    }
}

template <typename XT>
int launch_tiled_typed(const LinearGroup &g, cudaStream_t stream)
{
    uint32_t tiles = 0;
    for (uint32_t i = 0; i < g.count; i++) tiles += (g.seg[i].n + BN - 1) / BN;
    const dim3 grid(tiles, (g.m + BM - 1) / BM);
    if (g.glu) return launch(linear_tiled_kernel<XT, true>, grid, dim3(256), 0, stream, g);
    return launch(linear_tiled_kernel<XT, false>, grid, dim3(256), 0, stream, g);
}

int g_linear_force_tiled = 0;      // "linear.force_tiled"

}  // namespace

int set_linear_option(const char *name, long value)
{
    if (!__builtin_strcmp(name, "linear.force_tiled")) {
        g_linear_force_tiled = value ? 1 : 0;
        return MGQ_OK;
    }
    return fail(MGQ_ERR_NAME, "unknown option: %s", name);
}

int launch_linear_group(const LinearGroup &g, void *stream_v)
{
    cudaStream_t stream = static_cast<cudaStream_t>(stream_v);
    if (g.m == 0) return MGQ_OK;
    if (g.count == 0 || g.count > kMaxSegments || (g.glu && g.count != 1)) return fail(MGQ_ERR_SHAPE, "linear: %u layers", g.count);
    bool vec = true;
    for (uint32_t i = 0; i < g.count; i++) {
        const LinearSegment &s = g.seg[i];
        if (!s.a || !s.w || !s.out || (g.glu && (!s.w2 || !s.bias != !s.bias2))) return fail(MGQ_ERR_NULL, "linear: null operand");
        if (s.k == 0) return fail(MGQ_ERR_SHAPE, "linear: K is 0");
        vec = vec && s.k % 8 == 0 && reinterpret_cast<uintptr_t>(s.a) % 16 == 0 && reinterpret_cast<uintptr_t>(s.w) % 16 == 0 &&
              reinterpret_cast<uintptr_t>(s.w2) % 16 == 0;
    }
    if (g.m <= 8) return g.a_bf16 ? launch_gemv_typed<__nv_bfloat16>(g, vec, stream) : launch_gemv_typed<float>(g, vec, stream);
    if (g.a_bf16 && vec && !g_linear_force_tiled) return launch_linear_tc(g, stream_v);
    return g.a_bf16 ? launch_tiled_typed<__nv_bfloat16>(g, stream) : launch_tiled_typed<float>(g, stream);
}

}  // namespace mgq
