// Latent attention over a sliding window: the cache holds, per position, an RMS-normed latent of
// `rank` elements and one rotated key part of `rot_dim` elements shared by all heads.
//
// Absorbed form (few rows, and every f32 session): the query is folded through W_uk once,
//   score = (W_uk^T q_nope) . c + q_rot . k_rot,   o' = softmax . c,   o = W_uv o',
// so attention runs against the latents themselves and every head shares one key/value row.
//   latent_absorb_kernel   q' = scale * [W_uk^T q_nope | rotate(q_rot)]
//   latent_attend_kernel   CTA = 8 heads x one row x one slice of the window, 32 keys per tile,
//                          online softmax in f32; slices leave (max, sum, unnormalised o')
//   latent_out_kernel      merges the slices, applies W_uv and the output gate
// The ring cache is addressed by position % slots, so a sequence may be longer than the cache.
#include <algorithm>

#include "mgq_mixer.cuh"

namespace mgq {
namespace {

constexpr uint32_t kHeads = 8;             // heads per CTA in latent_attend_kernel
constexpr uint32_t kTile = 32;             // keys per tile
constexpr uint32_t kSliceKeys = 64;        // window positions per slice when the window is split
constexpr uint32_t kSplitRows = 16;        // at most this many rows split the window over CTAs

__device__ __forceinline__ void rotate_pair(float u, float v, uint32_t pos, float freq, float &ru, float &rv)
{
    float s, c;
    sincosf((float)pos * freq, &s, &c);
    ru = u * c - v * s;
    rv = v * c + u * s;
}

// ---------------------------------------------------------------- cache write: one CTA per row
template <typename CT>
__global__ void __launch_bounds__(128) latent_cache_kernel(const __grid_constant__ LatentCache a)
{
    __shared__ float s_part[4];
    const uint32_t t = threadIdx.x, row = blockIdx.x, width = a.rank + a.rot_dim, half = a.rot_dim / 2;
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t pos = a.pos[0] + row;
    const float *src = a.down + (size_t)row * width;
    CT *dst = static_cast<CT *>(a.cache) + (size_t)(pos % a.slots) * width;
    float ss = 0.f;
    for (uint32_t j = t; j < a.rank; j += 128) ss = fmaf(src[j], src[j], ss);
    ss = warp_sum(ss);
    if ((t & 31u) == 0) s_part[t >> 5] = ss;
    __syncthreads();
    const float r = 1.0f / sqrtf((s_part[0] + s_part[1] + s_part[2] + s_part[3]) / (float)a.rank + a.eps);
    for (uint32_t j = t; j < a.rank; j += 128) dst[j] = from_f32<CT>(src[j] * r * a.weight[j]);
    for (uint32_t i = t; i < half; i += 128) {
        float u, v;
        rotate_pair(src[a.rank + i], src[a.rank + half + i], pos, a.freq[i], u, v);
        dst[a.rank + i] = from_f32<CT>(u);
        dst[a.rank + half + i] = from_f32<CT>(v);
    }
}

// ---------------------------------------------------------------- q' = scale * [W_uk^T q_nope | rotate(q_rot)]
// CTA = head x AR rows x 64 rank columns: 32 column pairs x 8 slices of dim.
template <int AR>
__global__ void __launch_bounds__(256) latent_absorb_kernel(const __grid_constant__ LatentAttention a, float *qx)
{
    extern __shared__ float smem[];                      // [AR][dim] queries, then [8][AR][64] partials
    const uint32_t t = threadIdx.x, head = blockIdx.x, row0 = blockIdx.y * AR, c0 = blockIdx.z * 64, dim = a.dim, rot = a.rot_dim;
    const uint32_t qpitch = a.heads * (dim + rot), width = a.rank + rot, rows = min((uint32_t)AR, a.rows - row0);
    float *s_q = smem, *s_p = smem + AR * dim;
    pdl_launch_dependents();
    pdl_wait();
    for (uint32_t i = t; i < AR * dim; i += 256) {
        const uint32_t r = i / dim;
        s_q[i] = r < rows ? a.q[(size_t)(row0 + r) * qpitch + head * (dim + rot) + i - r * dim] * a.scale : 0.f;
    }
    __syncthreads();
    const uint32_t pair = t & 31u, slice = t >> 5, c = c0 + pair * 2;
    float acc[AR][2];
#pragma unroll
    for (int r = 0; r < AR; r++) acc[r][0] = acc[r][1] = 0.f;
    if (c < a.rank) {
        const bool two = c + 1 < a.rank;
        const bool wide = two && a.rank % 2 == 0;
        const __nv_bfloat16 *w = static_cast<const __nv_bfloat16 *>(a.uk) + (size_t)head * dim * a.rank + c;
#pragma unroll 8
        for (uint32_t d = slice; d < dim; d += 8) {
            float w0, w1;
            if (wide) {
                const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(w + (size_t)d * a.rank));
                w0 = f.x; w1 = f.y;
            } else {
                w0 = __bfloat162float(w[(size_t)d * a.rank]);
                w1 = two ? __bfloat162float(w[(size_t)d * a.rank + 1]) : 0.f;
            }
#pragma unroll
            for (int r = 0; r < AR; r++) {
                const float q = s_q[r * dim + d];
                acc[r][0] = fmaf(q, w0, acc[r][0]);
                acc[r][1] = fmaf(q, w1, acc[r][1]);
            }
        }
    }
#pragma unroll
    for (int r = 0; r < AR; r++) {
        s_p[(slice * AR + r) * 64 + pair * 2] = acc[r][0];
        s_p[(slice * AR + r) * 64 + pair * 2 + 1] = acc[r][1];
    }
    __syncthreads();
    for (uint32_t i = t; i < rows * 64; i += 256) {
        const uint32_t r = i / 64, j = i % 64;
        if (c0 + j >= a.rank) continue;
        float s = 0.f;
#pragma unroll
        for (int sl = 0; sl < 8; sl++) s += s_p[(sl * AR + r) * 64 + j];
        qx[((size_t)(row0 + r) * a.heads + head) * width + c0 + j] = s;
    }
    if (blockIdx.z == 0) {
        const uint32_t half = rot / 2, pos0 = a.pos[0] + row0;
        for (uint32_t i = t; i < rows * half; i += 256) {
            const uint32_t r = i / half, j = i - r * half;
            const float *q = a.q + (size_t)(row0 + r) * qpitch + head * (dim + rot) + dim;
            float u, v;
            rotate_pair(q[j], q[half + j], pos0 + r, a.freq[j], u, v);
            float *dst = qx + ((size_t)(row0 + r) * a.heads + head) * width + a.rank;
            dst[j] = u * a.scale;
            dst[half + j] = v * a.scale;
        }
    }
}

// ---------------------------------------------------------------- attention against the latents
__device__ __forceinline__ void load4(const float *p, float (&f)[4])
{
    const float4 v = *reinterpret_cast<const float4 *>(p);
    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
}
__device__ __forceinline__ void load4(const __nv_bfloat16 *p, float (&f)[4])
{
    const uint2 v = *reinterpret_cast<const uint2 *>(p);
    f[0] = __uint_as_float(v.x << 16); f[1] = __uint_as_float(v.x & 0xFFFF0000u);
    f[2] = __uint_as_float(v.y << 16); f[3] = __uint_as_float(v.y & 0xFFFF0000u);
}

__host__ __device__ inline uint32_t tile_pitch(uint32_t width) { return ((width + 3u) & ~3u) + 4u; }

// DPT: rank elements per thread (128 threads).  Partials: po [row][split][heads][rank], ml [row][split][heads][2].
template <typename CT, int DPT>
__global__ void __launch_bounds__(128) latent_attend_kernel(const __grid_constant__ LatentAttention a, const float *qx, float *po, float *ml)
{
    extern __shared__ __align__(16) float smem[];
    const uint32_t t = threadIdx.x, lane = t & 31u, warp = t >> 5, width = a.rank + a.rot_dim, pitch = tile_pitch(width);
    float *s_k = smem, *s_q = s_k + kTile * pitch;                       // [32][pitch], [8][pitch]
    __shared__ __align__(16) float s_p[kHeads][kTile];
    __shared__ float s_corr[kHeads];
    const uint32_t h0 = blockIdx.x * kHeads, split = blockIdx.y, splits = gridDim.y, row = blockIdx.z;
    const uint32_t heads = min(kHeads, a.heads - h0);
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t pos = a.pos[0] + row, lo = pos + 1 > a.window ? pos + 1 - a.window : 0u, total = pos + 1 - lo;
    const uint32_t per = ((total + splits - 1) / splits + kTile - 1) / kTile * kTile;
    const uint32_t k0 = min(lo + split * per, pos + 1), k1 = min(k0 + per, pos + 1);
    const size_t part = ((size_t)row * splits + split) * a.heads + h0;
    if (k0 >= k1) {
        if (t < heads) { ml[(part + t) * 2] = -INFINITY; ml[(part + t) * 2 + 1] = 0.f; }
        return;
    }
    for (uint32_t i = t; i < kHeads * pitch; i += 128) {
        const uint32_t h = i / pitch, j = i - h * pitch;
        s_q[i] = h < heads && j < width ? qx[((size_t)row * a.heads + h0 + h) * width + j] : 0.f;
    }
    for (uint32_t i = t; i < kTile * pitch; i += 128) s_k[i] = 0.f;      // the padding must stay finite
    __syncthreads();
    float acc[kHeads][DPT], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
    for (int h = 0; h < (int)kHeads; h++)
#pragma unroll
        for (int i = 0; i < DPT; i++) acc[h][i] = 0.f;
    const CT *cache = static_cast<const CT *>(a.cache);
    const bool vec = width % 4 == 0;
    for (uint32_t kt = k0; kt < k1; kt += kTile) {
        const uint32_t cnt = min(kTile, k1 - kt);
#pragma unroll 4
        for (uint32_t r = warp; r < kTile; r += 4) {
            if (r >= cnt) continue;
            const CT *src = cache + (size_t)((kt + r) % a.slots) * width;
            float *dst = s_k + r * pitch;
            if (vec) {
                for (uint32_t j = lane * 4; j < width; j += 128) {
                    float f[4];
                    load4(src + j, f);
                    *reinterpret_cast<float4 *>(dst + j) = make_float4(f[0], f[1], f[2], f[3]);
                }
            } else {
                for (uint32_t j = lane; j < width; j += 32) dst[j] = to_f32(src[j]);
            }
        }
        __syncthreads();
        // scores: lane = key, warp w = heads 2w and 2w + 1
        float s0 = 0.f, s1 = 0.f;
        const float *kr = s_k + lane * pitch, *q0 = s_q + (2 * warp) * pitch, *q1 = q0 + pitch;
#pragma unroll 4
        for (uint32_t d = 0; d < width; d += 4) {
            const float4 kv = *reinterpret_cast<const float4 *>(kr + d), x = *reinterpret_cast<const float4 *>(q0 + d),
                         y = *reinterpret_cast<const float4 *>(q1 + d);
            s0 = fmaf(kv.x, x.x, s0); s0 = fmaf(kv.y, x.y, s0); s0 = fmaf(kv.z, x.z, s0); s0 = fmaf(kv.w, x.w, s0);
            s1 = fmaf(kv.x, y.x, s1); s1 = fmaf(kv.y, y.y, s1); s1 = fmaf(kv.z, y.z, s1); s1 = fmaf(kv.w, y.w, s1);
        }
        float s[2] = {lane < cnt ? s0 : -INFINITY, lane < cnt ? s1 : -INFINITY};
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const float m_new = fmaxf(m[i], warp_max(s[i]));             // cnt >= 1: finite
            const float corr = expf(m[i] - m_new), p = expf(s[i] - m_new);
            l[i] = l[i] * corr + warp_sum(p);
            m[i] = m_new;
            s_p[2 * warp + i][lane] = p;
            if (lane == 0) s_corr[2 * warp + i] = corr;
        }
        __syncthreads();
#pragma unroll
        for (int h = 0; h < (int)kHeads; h++) {
            const float corr = s_corr[h];
#pragma unroll
            for (int i = 0; i < DPT; i++) acc[h][i] *= corr;
        }
        for (uint32_t k = 0; k < cnt; k += 4) {                          // rows beyond cnt: p = 0 and finite contents
            float kv[4][DPT];
#pragma unroll
            for (int u = 0; u < 4; u++)
#pragma unroll
                for (int i = 0; i < DPT; i++) {
                    const uint32_t d = t + 128u * i;
                    kv[u][i] = d < a.rank ? s_k[(k + u) * pitch + d] : 0.f;
                }
#pragma unroll
            for (int h = 0; h < (int)kHeads; h++) {
                const float4 p = *reinterpret_cast<const float4 *>(&s_p[h][k]);
#pragma unroll
                for (int i = 0; i < DPT; i++) {
                    acc[h][i] = fmaf(p.x, kv[0][i], acc[h][i]);
                    acc[h][i] = fmaf(p.y, kv[1][i], acc[h][i]);
                    acc[h][i] = fmaf(p.z, kv[2][i], acc[h][i]);
                    acc[h][i] = fmaf(p.w, kv[3][i], acc[h][i]);
                }
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int h = 0; h < (int)kHeads; h++) {
        if (h >= (int)heads) break;
#pragma unroll
        for (int i = 0; i < DPT; i++) {
            const uint32_t d = t + 128u * i;
            if (d < a.rank) po[(part + h) * a.rank + d] = acc[h][i];
        }
    }
    if (lane == 0) {
#pragma unroll
        for (int i = 0; i < 2; i++)
            if (2 * warp + i < heads) { ml[(part + 2 * warp + i) * 2] = m[i]; ml[(part + 2 * warp + i) * 2 + 1] = l[i]; }
    }
}

// ---------------------------------------------------------------- merge, W_uv, gate: CTA = row x head x 32 value dimensions
template <typename OT>
__global__ void __launch_bounds__(256) latent_out_kernel(const __grid_constant__ LatentAttention a, const float *po, const float *ml, uint32_t splits,
                                                         const __grid_constant__ HeadGate hg, OT *out)
{
    extern __shared__ __align__(16) float smem[];        // o' [rank], slice weights [splits]
    float *s_o = smem, *s_w = smem + ((a.rank + 3u) & ~3u);
    const uint32_t t = threadIdx.x, lane = t & 31u, warp = t >> 5, head = blockIdx.x, row = blockIdx.y, v0 = blockIdx.z * 32;
    const size_t part = (size_t)row * splits * a.heads + head;
    pdl_launch_dependents();
    pdl_wait();
    float m = -INFINITY, l = 0.f;
    for (uint32_t s = lane; s < splits; s += 32) m = fmaxf(m, ml[(part + (size_t)s * a.heads) * 2]);
    m = warp_max(m);
    for (uint32_t s = lane; s < splits; s += 32) {
        const float *p = ml + (part + (size_t)s * a.heads) * 2;
        const float w = expf(p[0] - m);
        if (warp == 0) s_w[s] = w;
        l = fmaf(p[1], w, l);
    }
    const float inv = 1.0f / warp_sum(l);
    __syncthreads();
    for (uint32_t d = t; d < a.rank; d += 256) {
        float s = 0.f;
#pragma unroll 4
        for (uint32_t i = 0; i < splits; i++) {
            const float w = s_w[i];
            if (w != 0.f) s = fmaf(po[(part + (size_t)i * a.heads) * a.rank + d], w, s);      // an empty slice has no partial
        }
        s_o[d] = s * inv;
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const uint32_t v = v0 + warp * 4 + i;
        if (v >= a.vdim) break;
        const __nv_bfloat16 *w = static_cast<const __nv_bfloat16 *>(a.uv) + ((size_t)head * a.vdim + v) * a.rank;
        float s = 0.f;
        if (a.rank % 8 == 0) {
            for (uint32_t c = lane * 8; c < a.rank; c += 256) {
                float wv[8];
                load8(w + c, wv);
                const float4 x = *reinterpret_cast<const float4 *>(s_o + c), y = *reinterpret_cast<const float4 *>(s_o + c + 4);
                s = fmaf(wv[0], x.x, s); s = fmaf(wv[1], x.y, s); s = fmaf(wv[2], x.z, s); s = fmaf(wv[3], x.w, s);
                s = fmaf(wv[4], y.x, s); s = fmaf(wv[5], y.y, s); s = fmaf(wv[6], y.z, s); s = fmaf(wv[7], y.w, s);
            }
        } else {
            for (uint32_t c = lane; c < a.rank; c += 32) s = fmaf(__bfloat162float(w[c]), s_o[c], s);
        }
        s = warp_sum(s);
        if (lane == 0) {
            const size_t o = ((size_t)row * a.heads + head) * a.vdim + v;
            if (hg.gate) {
                const float g = hg.gate[o], sg = sigmoid_f(g);
                s *= hg.silu ? g * sg : sg;
            }
            out[o] = from_f32<OT>(s);
        }
    }
}

uint32_t window_splits(uint32_t rows, uint32_t window) { return rows <= kSplitRows ? (window + kSliceKeys - 1) / kSliceKeys : 1u; }

template <typename CT, int DPT>
int launch_attend_dpt(const LatentAttention &a, const float *qx, float *po, float *ml, uint32_t splits, cudaStream_t st)
{
    const size_t smem = (size_t)(kTile + kHeads) * tile_pitch(a.rank + a.rot_dim) * sizeof(float);
    if (int rc = allow_smem(latent_attend_kernel<CT, DPT>, smem)) return rc;
    return launch(latent_attend_kernel<CT, DPT>, dim3((a.heads + kHeads - 1) / kHeads, splits, a.rows), dim3(128), smem, st, a, qx, po, ml);
}

template <typename CT>
int launch_attend(const LatentAttention &a, const float *qx, float *po, float *ml, uint32_t splits, cudaStream_t st)
{
    if (a.rank <= 128) return launch_attend_dpt<CT, 1>(a, qx, po, ml, splits, st);
    if (a.rank <= 256) return launch_attend_dpt<CT, 2>(a, qx, po, ml, splits, st);
    if (a.rank <= 512) return launch_attend_dpt<CT, 4>(a, qx, po, ml, splits, st);
    return launch_attend_dpt<CT, 8>(a, qx, po, ml, splits, st);
}

template <int AR>
int launch_absorb(const LatentAttention &a, float *qx, cudaStream_t st)
{
    const size_t smem = (size_t)AR * (a.dim + 8 * 64) * sizeof(float);
    if (int rc = allow_smem(latent_absorb_kernel<AR>, smem)) return rc;
    return launch(latent_absorb_kernel<AR>, dim3(a.heads, (a.rows + AR - 1) / AR, (a.rank + 63) / 64), dim3(256), smem, st, a, qx);
}

template <typename OT>
int launch_out(const LatentAttention &a, const float *po, const float *ml, uint32_t splits, const HeadGate &hg, void *out, cudaStream_t st)
{
    const size_t smem = (size_t)(((a.rank + 3) & ~3u) + splits) * sizeof(float);
    return launch(latent_out_kernel<OT>, dim3(a.heads, a.rows, (a.vdim + 31) / 32), dim3(256), smem, st, a, po, ml, splits, hg, static_cast<OT *>(out));
}

size_t align256(size_t n) { return (n + 255) & ~(size_t)255; }

size_t absorbed_bytes(uint32_t max_rows, uint32_t heads, uint32_t rot_dim, uint32_t rank, uint32_t window)
{
    const size_t parts = std::max<size_t>(max_rows, (size_t)std::min(max_rows, kSplitRows) * window_splits(1, window));
    return align256((size_t)max_rows * heads * (rank + rot_dim) * 4) + align256(parts * heads * rank * 4) + align256(parts * heads * 8);
}

}  // namespace

int launch_latent_cache_write(const LatentCache &a, void *stream)
{
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (a.rows > a.slots) return fail(MGQ_ERR_SHAPE, "latent cache: %u rows into a ring of %u", a.rows, a.slots);
    if (a.cache_bf16) return launch(latent_cache_kernel<__nv_bfloat16>, dim3(a.rows), dim3(128), 0, st, a);
    return launch(latent_cache_kernel<float>, dim3(a.rows), dim3(128), 0, st, a);
}

size_t latent_attention_workspace(uint32_t max_rows, uint32_t heads, uint32_t dim, uint32_t rot_dim, uint32_t vdim, uint32_t rank, uint32_t slots,
                                  uint32_t window, bool cache_bf16)
{
    (void)dim; (void)vdim; (void)slots; (void)cache_bf16;
    return absorbed_bytes(max_rows, heads, rot_dim, rank, window);
}

int launch_latent_attention(const LatentAttention &a, void *stream)
{
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (a.rank > 1024) return fail(MGQ_ERR_SHAPE, "latent attention: a latent of %u elements (at most 1024)", a.rank);
    if (a.rows > a.slots || a.window + a.rows - 1 > a.slots) return fail(MGQ_ERR_SHAPE, "latent attention: %u rows and a window of %u need more than %u cache rows", a.rows, a.window, a.slots);
    const uint32_t width = a.rank + a.rot_dim, splits = window_splits(a.rows, a.window);
    float *qx = static_cast<float *>(a.workspace);
    uint8_t *at = static_cast<uint8_t *>(a.workspace) + align256((size_t)a.rows * a.heads * width * 4);
    float *po = reinterpret_cast<float *>(at);
    float *ml = reinterpret_cast<float *>(at + align256((size_t)a.rows * splits * a.heads * a.rank * 4));
    if (int rc = a.rows == 1 ? launch_absorb<1>(a, qx, st) : launch_absorb<8>(a, qx, st)) return rc;
    if (int rc = a.cache_bf16 ? launch_attend<__nv_bfloat16>(a, qx, po, ml, splits, st) : launch_attend<float>(a, qx, po, ml, splits, st)) return rc;
    const HeadGate none{};
    const HeadGate &hg = a.gate ? *a.gate : none;
    void *out = a.gate ? a.gate->out : a.o;
    if (a.gate && a.gate->out_bf16) return launch_out<__nv_bfloat16>(a, po, ml, splits, hg, out, st);
    return launch_out<float>(a, po, ml, splits, hg, out, st);
}

}  // namespace mgq
