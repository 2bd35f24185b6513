// Latent attention over a sliding window: the cache holds, per position, an RMS-normed latent of
// `rank` elements and one rotated key part of `rot_dim` elements shared by all heads.
//
// Absorbed form (few rows, and every f32 session; many rows: mgq_prefill_attention.cu): the query is folded through W_uk once,
//   score = (W_uk^T q_nope) . c + q_rot . k_rot,   o' = softmax . c,   o = W_uv o',
// so attention runs against the latents themselves and every head shares one key/value row.
//   latent_absorb_kernel   q' = scale * [W_uk^T q_nope | rotate(q_rot)]
//   latent_attend_kernel   CTA = 8 heads (a warp each) x one row x one slice of the window, 32 keys per tile,
//                          online softmax in f32; slices leave (max, sum, unnormalised o')
//   latent_attend_mma_kernel   the same for bf16 caches: 16 heads x 64 keys on the tensor cores; the f32
//                          query and the f32 weights enter as sums of two bf16
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
    for (uint32_t d = t; d < dim; d += 256)              // weights are immutable: towards L2 before the wait
        asm volatile("prefetch.global.L2 [%0];" ::"l"(static_cast<const __nv_bfloat16 *>(a.uk) + ((size_t)head * dim + d) * a.rank + c0));
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
#pragma unroll(AR == 1 ? 16 : 8)
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
// Shared-memory row pitch in elements: 16-byte pieces of consecutive rows fall into different banks.
template <typename CT> __host__ __device__ inline uint32_t key_pitch(uint32_t width)
{
    constexpr uint32_t per = 16 / sizeof(CT);
    const uint32_t pieces = (width + per - 1) / per;
    return (pieces | 1u) * per;
}
__host__ __device__ inline uint32_t query_pitch(uint32_t width) { return (width + 7u) & ~7u; }

__device__ __forceinline__ void unpack_piece(const float *p, float (&f)[4])
{
    const float4 v = *reinterpret_cast<const float4 *>(p);
    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
}
__device__ __forceinline__ void unpack_piece(const __nv_bfloat16 *p, float (&f)[8]) { unpack8(*reinterpret_cast<const uint4 *>(p), f); }

__device__ __forceinline__ void cp_async16(void *smem, const void *gmem)
{
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((unsigned)__cvta_generic_to_shared(smem)), "l"(gmem) : "memory");
}

// DPT: pairs of rank elements per thread (256 threads).  A warp scores one head against a tile of 32
// keys (lane = key), then every thread adds its rank elements for all 8 heads.
// Partials: po [row][split][heads][rank], ml [row][split][heads][2].
template <typename CT, int DPT>
__global__ void __launch_bounds__(256) latent_attend_kernel(const __grid_constant__ LatentAttention a, const float *qx, float *po, float *ml)
{
    constexpr uint32_t PER = 16 / sizeof(CT);
    extern __shared__ __align__(16) float smem[];
    const uint32_t t = threadIdx.x, lane = t & 31u, warp = t >> 5, width = a.rank + a.rot_dim, kp = key_pitch<CT>(width), qp = query_pitch(width);
    float *s_q = smem;                                                   // [8][qp]
    CT *s_k = reinterpret_cast<CT *>(smem + kHeads * qp);                // [32][kp]
    __shared__ __align__(16) float s_p[kHeads][kTile];
    __shared__ float s_corr[kHeads];
    const uint32_t h0 = blockIdx.x * kHeads, split = blockIdx.y, splits = gridDim.y, row = blockIdx.z;
    const uint32_t heads = min(kHeads, a.heads - h0);
    pdl_launch_dependents();
    // the padding behind a row must stay finite
    for (uint32_t i = t; i < kTile * (kp - width); i += 256) s_k[(i / (kp - width)) * kp + width + i % (kp - width)] = from_f32<CT>(0.f);
    pdl_wait();
    const uint32_t pos = a.pos[0] + row, lo = pos + 1 > a.window ? pos + 1 - a.window : 0u, total = pos + 1 - lo;
    const uint32_t per = ((total + splits - 1) / splits + kTile - 1) / kTile * kTile;
    const uint32_t k0 = min(lo + split * per, pos + 1), k1 = min(k0 + per, pos + 1);
    const size_t part = ((size_t)row * splits + split) * a.heads + h0;
    if (k0 >= k1) {
        if (t < heads) { ml[(part + t) * 2] = -INFINITY; ml[(part + t) * 2 + 1] = 0.f; }
        return;
    }
    const CT *cache = static_cast<const CT *>(a.cache);
    const bool vec = width % PER == 0;
    auto stage = [&](uint32_t kt) {
#pragma unroll
        for (uint32_t r = warp; r < kTile; r += 8) {
            if (kt + r < k1) {
                const CT *src = cache + (size_t)((kt + r) % a.slots) * width;
                CT *dst = s_k + r * kp;
                if (vec) {
                    for (uint32_t j = lane * PER; j < width; j += 32 * PER) cp_async16(dst + j, src + j);
                } else {
                    for (uint32_t j = lane; j < width; j += 32) dst[j] = src[j];
                }
            } else {
                for (uint32_t j = lane; j < width; j += 32) s_k[r * kp + j] = from_f32<CT>(0.f);
            }
        }
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };
    stage(k0);
    const float *qsrc = qx + ((size_t)row * a.heads + h0) * width;
    if (width % 4 == 0) {
        for (uint32_t h = warp; h < kHeads; h += 8)
            for (uint32_t j = lane * 4; j < qp; j += 128)
                *reinterpret_cast<float4 *>(s_q + h * qp + j) = h < heads && j < width ? *reinterpret_cast<const float4 *>(qsrc + h * width + j) : make_float4(0.f, 0.f, 0.f, 0.f);
    } else {
        for (uint32_t h = warp; h < kHeads; h += 8)
            for (uint32_t j = lane; j < qp; j += 32) s_q[h * qp + j] = h < heads && j < width ? qsrc[h * width + j] : 0.f;
    }
    float acc[kHeads][2 * DPT], m = -INFINITY, l = 0.f;
#pragma unroll
    for (int h = 0; h < (int)kHeads; h++)
#pragma unroll
        for (int i = 0; i < 2 * DPT; i++) acc[h][i] = 0.f;
    for (uint32_t kt = k0; kt < k1; kt += kTile) {
        asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        __syncthreads();
        float s4[4] = {0.f, 0.f, 0.f, 0.f};
        const CT *kr = s_k + lane * kp;
        const float *q = s_q + warp * qp;
#pragma unroll 4
        for (uint32_t d = 0; d < width; d += PER) {                      // the query is zero beyond width
            float kv[PER];
            unpack_piece(kr + d, kv);
#pragma unroll
            for (int j = 0; j < (int)PER; j += 4) {
                const float4 x = *reinterpret_cast<const float4 *>(q + d + j);
                s4[0] = fmaf(kv[j], x.x, s4[0]); s4[1] = fmaf(kv[j + 1], x.y, s4[1]);
                s4[2] = fmaf(kv[j + 2], x.z, s4[2]); s4[3] = fmaf(kv[j + 3], x.w, s4[3]);
            }
        }
        const float s = kt + lane < k1 ? (s4[0] + s4[1]) + (s4[2] + s4[3]) : -INFINITY;
        const float m_new = fmaxf(m, warp_max(s));                       // at least one key: finite
        const float corr = expf(m - m_new), p = expf(s - m_new);
        l = l * corr + warp_sum(p);
        m = m_new;
        s_p[warp][lane] = p;
        if (lane == 0) s_corr[warp] = corr;
        __syncthreads();
#pragma unroll
        for (int h = 0; h < (int)kHeads; h++) {
            const float c = s_corr[h];
#pragma unroll
            for (int i = 0; i < 2 * DPT; i++) acc[h][i] *= c;
        }
#pragma unroll 2
        for (uint32_t k = 0; k < kTile; k += 4) {
            float kv[4][2 * DPT];
#pragma unroll
            for (int u = 0; u < 4; u++)
#pragma unroll
                for (int i = 0; i < DPT; i++) {
                    const uint32_t d = 2 * (t + 256u * i);               // an odd rank reads one element of the rotated part, never stored
                    kv[u][2 * i] = d < a.rank ? to_f32(s_k[(k + u) * kp + d]) : 0.f;
                    kv[u][2 * i + 1] = d < a.rank ? to_f32(s_k[(k + u) * kp + d + 1]) : 0.f;
                }
#pragma unroll
            for (int h = 0; h < (int)kHeads; h++) {
                const float4 p4 = *reinterpret_cast<const float4 *>(&s_p[h][k]);
#pragma unroll
                for (int i = 0; i < 2 * DPT; i++) {
                    acc[h][i] = fmaf(p4.x, kv[0][i], acc[h][i]);
                    acc[h][i] = fmaf(p4.y, kv[1][i], acc[h][i]);
                    acc[h][i] = fmaf(p4.z, kv[2][i], acc[h][i]);
                    acc[h][i] = fmaf(p4.w, kv[3][i], acc[h][i]);
                }
            }
        }
        __syncthreads();
        if (kt + kTile < k1) stage(kt + kTile);
    }
#pragma unroll
    for (int h = 0; h < (int)kHeads; h++) {
        if (h >= (int)heads) break;
#pragma unroll
        for (int i = 0; i < DPT; i++) {
            const uint32_t d = 2 * (t + 256u * i);
            float *dst = po + (part + h) * a.rank + d;
            if (d < a.rank) dst[0] = acc[h][2 * i];
            if (d + 1 < a.rank) dst[1] = acc[h][2 * i + 1];
        }
    }
    if (lane == 0 && warp < heads) { ml[(part + warp) * 2] = m; ml[(part + warp) * 2 + 1] = l; }
}

// ---------------------------------------------------------------- the same on the tensor cores (bf16 cache, sizes in multiples of 8)
__device__ __forceinline__ uint32_t smem_addr(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldmatrix4(uint32_t addr, uint32_t (&r)[4])
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldmatrix2(uint32_t addr, uint32_t (&r)[2])
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0, %1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldmatrix4_t(uint32_t addr, uint32_t (&r)[4])
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1)
{
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

constexpr uint32_t kMmaHeads = 16, kMmaTile = 64;
__host__ __device__ inline uint32_t mma_pitch(uint32_t width) { return (width + 15u) / 16u * 16u + 8u; }      // an odd number of 16-byte pieces
inline size_t mma_smem(uint32_t width) { return ((size_t)kMmaTile + 2 * kMmaHeads) * mma_pitch(width) * 2; }

// NT: 16-column groups of the latent per warp (8 warps): rank <= 128 * NT.
template <int NT>
__global__ void __launch_bounds__(256) latent_attend_mma_kernel(const __grid_constant__ LatentAttention a, const float *qx, float *po, float *ml)
{
    extern __shared__ __align__(16) __nv_bfloat16 sm[];
    __shared__ float s_s[kMmaHeads][kMmaTile + 1], s_corr[kMmaHeads];
    __shared__ __align__(16) __nv_bfloat16 s_p[2][kMmaHeads][kMmaTile + 8];
    const uint32_t t = threadIdx.x, lane = t & 31u, warp = t >> 5, width = a.rank + a.rot_dim, pitch = mma_pitch(width), k16 = (width + 15u) / 16u;
    __nv_bfloat16 *s_k = sm, *s_hi = s_k + kMmaTile * pitch, *s_lo = s_hi + kMmaHeads * pitch;
    const uint32_t h0 = blockIdx.x * kMmaHeads, split = blockIdx.y, splits = gridDim.y, row = blockIdx.z;
    const uint32_t heads = min(kMmaHeads, a.heads - h0);
    pdl_launch_dependents();
    const uint32_t pad = k16 * 16 - width;               // zero columns behind the rows, so that garbage never meets a zero
    for (uint32_t i = t; i < kMmaTile * pad; i += 256) s_k[(i / pad) * pitch + width + i % pad] = __float2bfloat16_rn(0.f);
    pdl_wait();
    const uint32_t pos = a.pos[0] + row, lo = pos + 1 > a.window ? pos + 1 - a.window : 0u, total = pos + 1 - lo;
    const uint32_t per = ((total + splits - 1) / splits + kMmaTile - 1) / kMmaTile * kMmaTile;
    const uint32_t k0 = min(lo + split * per, pos + 1), k1 = min(k0 + per, pos + 1);
    const size_t part = ((size_t)row * splits + split) * a.heads + h0;
    if (k0 >= k1) {
        if (t < heads) { ml[(part + t) * 2] = -INFINITY; ml[(part + t) * 2 + 1] = 0.f; }
        return;
    }
    const __nv_bfloat16 *cache = static_cast<const __nv_bfloat16 *>(a.cache);
    auto stage = [&](uint32_t kt) {
#pragma unroll
        for (uint32_t r = warp; r < kMmaTile; r += 8) {                   // beyond the last key: a valid row, masked below
            const __nv_bfloat16 *src = cache + (size_t)(min(kt + r, k1 - 1u) % a.slots) * width;
            for (uint32_t j = lane * 8; j < width; j += 256) cp_async16(s_k + r * pitch + j, src + j);
        }
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };
    stage(k0);
    const float *qsrc = qx + ((size_t)row * a.heads + h0) * width;
    for (uint32_t h = warp; h < kMmaHeads; h += 8)
#pragma unroll 4
        for (uint32_t j = lane * 2; j < k16 * 16; j += 64) {
            const float2 q = h < heads && j < width ? *reinterpret_cast<const float2 *>(qsrc + h * width + j) : make_float2(0.f, 0.f);
            const __nv_bfloat162 hi = __floats2bfloat162_rn(q.x, q.y);
            const float2 f = __bfloat1622float2(hi);
            *reinterpret_cast<__nv_bfloat162 *>(s_hi + h * pitch + j) = hi;
            *reinterpret_cast<__nv_bfloat162 *>(s_lo + h * pitch + j) = __floats2bfloat162_rn(q.x - f.x, q.y - f.y);
        }
    float o[2 * NT][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};      // m, l: heads 2 * warp, 2 * warp + 1
#pragma unroll
    for (int n = 0; n < 2 * NT; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) o[n][e] = 0.f;
    const uint32_t a_off = (((lane & 7u) + ((lane >> 3) & 1u) * 8) * pitch + (lane >> 4) * 8) * 2;
    const uint32_t hi_addr = smem_addr(s_hi) + a_off, lo_addr = smem_addr(s_lo) + a_off;
    const uint32_t b_addr = smem_addr(s_k + (warp * 8 + (lane & 7u)) * pitch + ((lane >> 3) & 1u) * 8);
    const uint32_t v_addr = smem_addr(s_k) + (((lane & 7u) + ((lane >> 3) & 1u) * 8) * pitch + (lane >> 4) * 8) * 2;
    const uint32_t p_off = (((lane & 7u) + ((lane >> 3) & 1u) * 8) * (kMmaTile + 8) + (lane >> 4) * 8) * 2;
    for (uint32_t kt = k0; kt < k1; kt += kMmaTile) {
        asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        __syncthreads();
        float s_hi_acc[4] = {0.f, 0.f, 0.f, 0.f}, s_lo_acc[4] = {0.f, 0.f, 0.f, 0.f};       // warp w: keys 8w .. 8w + 7
#pragma unroll 4
        for (uint32_t kk = 0; kk < k16; kk++) {
            uint32_t ah[4], al[4], b[2];
            ldmatrix4(hi_addr + kk * 32, ah);
            ldmatrix4(lo_addr + kk * 32, al);
            ldmatrix2(b_addr + kk * 32, b);
            mma16816(s_hi_acc, ah, b[0], b[1]);
            mma16816(s_lo_acc, al, b[0], b[1]);
        }
#pragma unroll
        for (int e = 0; e < 4; e++) s_s[lane / 4 + (e >> 1) * 8][warp * 8 + (lane & 3u) * 2 + (e & 1)] = s_hi_acc[e] + s_lo_acc[e];
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const uint32_t h = warp * 2 + i;
            const float x = kt + lane < k1 ? s_s[h][lane] : -INFINITY, y = kt + lane + 32 < k1 ? s_s[h][lane + 32] : -INFINITY;
            const float m_new = fmaxf(m[i], warp_max(fmaxf(x, y)));      // at least one key: finite
            const float corr = expf(m[i] - m_new), px = expf(x - m_new), py = expf(y - m_new);
            l[i] = l[i] * corr + warp_sum(px + py);
            m[i] = m_new;
            const __nv_bfloat16 hx = __float2bfloat16_rn(px), hy = __float2bfloat16_rn(py);
            s_p[0][h][lane] = hx;
            s_p[0][h][lane + 32] = hy;
            s_p[1][h][lane] = __float2bfloat16_rn(px - __bfloat162float(hx));
            s_p[1][h][lane + 32] = __float2bfloat16_rn(py - __bfloat162float(hy));
            if (lane == 0) s_corr[h] = corr;
        }
        __syncthreads();
        const float c0 = s_corr[lane / 4], c1 = s_corr[lane / 4 + 8];
#pragma unroll
        for (int n = 0; n < 2 * NT; n++) { o[n][0] *= c0; o[n][1] *= c0; o[n][2] *= c1; o[n][3] *= c1; }
#pragma unroll
        for (int kk = 0; kk < (int)kMmaTile / 16; kk++) {
            uint32_t ph[4], pl[4];
            ldmatrix4(smem_addr(s_p[0]) + p_off + kk * 32, ph);
            ldmatrix4(smem_addr(s_p[1]) + p_off + kk * 32, pl);
#pragma unroll
            for (int n = 0; n < NT; n++) {
                const uint32_t col = (warp * NT + n) * 16;
                if (col >= a.rank) break;
                uint32_t b[4];
                ldmatrix4_t(v_addr + (kk * 16 * pitch + col) * 2, b);
                mma16816(o[2 * n], ph, b[0], b[1]);
                mma16816(o[2 * n + 1], ph, b[2], b[3]);
                mma16816(o[2 * n], pl, b[0], b[1]);
                mma16816(o[2 * n + 1], pl, b[2], b[3]);
            }
        }
        __syncthreads();
        if (kt + kMmaTile < k1) stage(kt + kMmaTile);
    }
#pragma unroll
    for (int n = 0; n < 2 * NT; n++) {
        const uint32_t col = (warp * NT + n / 2) * 16 + (n & 1) * 8 + (lane & 3u) * 2;
        if (col >= a.rank) break;                        // rank % 8 == 0: pairs never straddle it
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const uint32_t h = lane / 4 + 8 * i;
            if (h < heads) *reinterpret_cast<float2 *>(po + (part + h) * a.rank + col) = make_float2(o[n][2 * i], o[n][2 * i + 1]);
        }
    }
#pragma unroll
    for (int i = 0; i < 2; i++)
        if (lane == 0 && warp * 2 + i < heads) { ml[(part + warp * 2 + i) * 2] = m[i]; ml[(part + warp * 2 + i) * 2 + 1] = l[i]; }
}

// ---------------------------------------------------------------- merge, W_uv, gate: CTA = row x head x 64 value dimensions
constexpr uint32_t kOutThreads = 512, kOutDims = 64;

template <typename OT>
__global__ void __launch_bounds__(kOutThreads) latent_out_kernel(const __grid_constant__ LatentAttention a, const float *po, const float *ml, uint32_t splits,
                                                                 const __grid_constant__ HeadGate hg, OT *out)
{
    extern __shared__ __align__(16) float smem[];        // o' [rank], slice weights [splits]
    float *s_o = smem, *s_w = smem + ((a.rank + 3u) & ~3u);
    const uint32_t t = threadIdx.x, lane = t & 31u, warp = t >> 5, head = blockIdx.x, row = blockIdx.y, v0 = blockIdx.z * kOutDims + warp * 4;
    const size_t part = (size_t)row * splits * a.heads + head;
    const __nv_bfloat16 *uv = static_cast<const __nv_bfloat16 *>(a.uv) + (size_t)head * a.vdim * a.rank;
    pdl_launch_dependents();
#pragma unroll
    for (int i = 0; i < 4; i++)                          // weights are immutable: towards L2 before the wait
        if (v0 + i < a.vdim && lane * 64u < a.rank) asm volatile("prefetch.global.L2 [%0];" ::"l"(uv + (size_t)(v0 + i) * a.rank + lane * 64u));
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
    for (uint32_t d = t; d < a.rank; d += kOutThreads) {
        const float *src = po + part * a.rank + d;
        const size_t step = (size_t)a.heads * a.rank;
        float s = 0.f;
#pragma unroll 16
        for (uint32_t i = 0; i < splits; i++) {
            const float w = s_w[i];
            s = w != 0.f ? fmaf(src[i * step], w, s) : s;              // an empty slice has no partial
        }
        s_o[d] = s * inv;
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const uint32_t v = v0 + i;
        if (v >= a.vdim) break;
        const __nv_bfloat16 *w = uv + (size_t)v * a.rank;
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
    const uint32_t width = a.rank + a.rot_dim;
    const size_t smem = (size_t)kHeads * query_pitch(width) * sizeof(float) + (size_t)kTile * key_pitch<CT>(width) * sizeof(CT);
    if (int rc = allow_smem(latent_attend_kernel<CT, DPT>, smem)) return rc;
    return launch(latent_attend_kernel<CT, DPT>, dim3((a.heads + kHeads - 1) / kHeads, splits, a.rows), dim3(256), smem, st, a, qx, po, ml);
}

template <typename CT>
int launch_attend(const LatentAttention &a, const float *qx, float *po, float *ml, uint32_t splits, cudaStream_t st)
{
    if (a.rank <= 512) return launch_attend_dpt<CT, 1>(a, qx, po, ml, splits, st);
    return launch_attend_dpt<CT, 2>(a, qx, po, ml, splits, st);
}

template <int NT>
int launch_mma_nt(const LatentAttention &a, const float *qx, float *po, float *ml, uint32_t splits, cudaStream_t st)
{
    const size_t smem = mma_smem(a.rank + a.rot_dim);
    if (int rc = allow_smem(latent_attend_mma_kernel<NT>, smem)) return rc;
    return launch(latent_attend_mma_kernel<NT>, dim3((a.heads + kMmaHeads - 1) / kMmaHeads, splits, a.rows), dim3(256), smem, st, a, qx, po, ml);
}

int launch_mma(const LatentAttention &a, const float *qx, float *po, float *ml, uint32_t splits, cudaStream_t st)
{
    if (a.rank <= 128) return launch_mma_nt<1>(a, qx, po, ml, splits, st);
    if (a.rank <= 256) return launch_mma_nt<2>(a, qx, po, ml, splits, st);
    if (a.rank <= 512) return launch_mma_nt<4>(a, qx, po, ml, splits, st);
    return launch_mma_nt<8>(a, qx, po, ml, splits, st);
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
    if (int rc = allow_smem(latent_out_kernel<OT>, smem)) return rc;
    return launch(latent_out_kernel<OT>, dim3(a.heads, a.rows, (a.vdim + kOutDims - 1) / kOutDims), dim3(kOutThreads), smem, st, a, po, ml, splits, hg, static_cast<OT *>(out));
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
    if (!latent_prefill_eligible(dim, rot_dim, vdim, rank, cache_bf16)) return absorbed_bytes(max_rows, heads, rot_dim, rank, window);
    const size_t few = absorbed_bytes(std::min(max_rows, kPrefillRows - 1), heads, rot_dim, rank, window);
    return max_rows < kPrefillRows ? few : std::max(few, latent_prefill_workspace(heads, dim, rot_dim, vdim, slots));
}

int launch_latent_attention(const LatentAttention &a, void *stream)
{
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (a.rank > 1024) return fail(MGQ_ERR_SHAPE, "latent attention: a latent of %u elements (at most 1024)", a.rank);
    if (a.rows > a.slots || a.window + a.rows - 1 > a.slots) return fail(MGQ_ERR_SHAPE, "latent attention: %u rows and a window of %u need more than %u cache rows", a.rows, a.window, a.slots);
    if (a.rows >= kPrefillRows && latent_prefill_eligible(a.dim, a.rot_dim, a.vdim, a.rank, a.cache_bf16)) return launch_latent_prefill(a, stream);
    const uint32_t width = a.rank + a.rot_dim, splits = window_splits(a.rows, a.window);
    float *qx = static_cast<float *>(a.workspace);
    uint8_t *at = static_cast<uint8_t *>(a.workspace) + align256((size_t)a.rows * a.heads * width * 4);
    float *po = reinterpret_cast<float *>(at);
    float *ml = reinterpret_cast<float *>(at + align256((size_t)a.rows * splits * a.heads * a.rank * 4));
    if (int rc = a.rows == 1 ? launch_absorb<1>(a, qx, st) : launch_absorb<8>(a, qx, st)) return rc;
    const bool mma = a.cache_bf16 && a.rank % 8 == 0 && a.rot_dim % 8 == 0 && mma_smem(width) <= 210 * 1024;
    if (int rc = mma ? launch_mma(a, qx, po, ml, splits, st) : a.cache_bf16 ? launch_attend<__nv_bfloat16>(a, qx, po, ml, splits, st) : launch_attend<float>(a, qx, po, ml, splits, st)) return rc;
    const HeadGate none{};
    const HeadGate &hg = a.gate ? *a.gate : none;
    void *out = a.gate ? a.gate->out : a.o;
    if (a.gate && a.gate->out_bf16) return launch_out<__nv_bfloat16>(a, po, ml, splits, hg, out, st);
    return launch_out<float>(a, po, ml, splits, hg, out, st);
}

}  // namespace mgq
