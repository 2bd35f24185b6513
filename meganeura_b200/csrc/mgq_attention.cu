// Causal softmax attention with grouped key / value heads, and what stands between the projections and it.
//
// Caches are [slots, kv_heads * dim] and [slots, kv_heads * vdim], f32 or f16 (clamped to its range; 11
// significant bits).  The unit of the kernels for few rows is a PAIR (row, query head of one key / value
// head): the pairs of a key / value head share its keys, whether they are several heads of one decoded
// token or several tokens of a short portion.
//   attention_mma_kernel   f16 caches, sizes in multiples of 8: CTA = 16 pairs x one slice of the keys, on the
//                          tensor cores; every warp runs its own online softmax over its 16 keys of a tile
//   attention_kernel       any size, f32 or f16: CTA = 8 pairs (a warp each) x one slice, f32 arithmetic
//   attention_merge_kernel puts the slices together and applies the output gate
// Many rows over f16 caches: mgq_prefill_attention.cu.  Scores, maxima and sums are f32 (base-2 exponentials);
// queries and weights enter the tensor-core products as f16 in all forms, so it hardly matters how a prompt is cut.
#include <algorithm>

#include "mgq_mixer.cuh"

namespace mgq {
namespace {

constexpr float kLog2e = 1.4426950408889634f;

// ---------------------------------------------------------------- query temperature, caches, both with the norms
__device__ __forceinline__ float temperature(uint32_t p, float coef, float every)
{
    return fmaf(coef, logf(floorf((float)(p + 1u) / every) + 1.0f), 1.0f);
}

__global__ void query_temperature_kernel(const float *x, const uint32_t *pos, float *out, uint32_t rows, uint32_t cols, float coef, float every)
{
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    pdl_launch_dependents();
    pdl_wait();
    if (i >= (size_t)rows * cols) return;
    out[i] = x[i] * temperature(pos[0] + (uint32_t)(i / cols), coef, every);
}

template <typename CT>
__global__ void cache_append_kernel(const float *x, CT *cache, const uint32_t *pos, uint32_t rows, uint32_t cols, uint32_t slots)
{
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    pdl_launch_dependents();
    pdl_wait();
    if (i >= (size_t)rows * cols) return;
    const uint32_t row = (uint32_t)(i / cols), slot = pos[0] + row;
    if (slot < slots) cache[(size_t)slot * cols + (i - (size_t)row * cols)] = from_f32<CT>(x[i]);
}

__device__ __forceinline__ void store4(float *p, const float4 &x) { *reinterpret_cast<float4 *>(p) = x; }
__device__ __forceinline__ void store4(__half *p, const float4 &x)
{
    const __half2 a = __halves2half2(from_f32<__half>(x.x), from_f32<__half>(x.y)), b = __halves2half2(from_f32<__half>(x.z), from_f32<__half>(x.w));
    *reinterpret_cast<uint2 *>(p) = make_uint2(*reinterpret_cast<const uint32_t *>(&a), *reinterpret_cast<const uint32_t *>(&b));
}

// CTA = row; widths in multiples of 4, at most 1024 * NV.
template <typename CT, int NV>
__global__ void __launch_bounds__(256) attention_inputs_vec_kernel(const __grid_constant__ AttentionInputs a)
{
    __shared__ float s_part[2][8];
    const uint32_t t = threadIdx.x, row = blockIdx.x, nq = a.q_cols / 4, nk = a.k_cols / 4, nv = a.v_cols / 4;
    float4 q[NV], k[NV], v[NV];
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t p = a.pos[0] + row;
    const float4 *qs = reinterpret_cast<const float4 *>(a.q + (size_t)row * a.q_cols), *ks = reinterpret_cast<const float4 *>(a.k + (size_t)row * a.k_cols),
                 *vs = reinterpret_cast<const float4 *>(a.v + (size_t)row * a.v_cols);
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    float sq = 0.f, sk = 0.f;
#pragma unroll
    for (int i = 0; i < NV; i++) {
        const uint32_t j = t + 256u * i;
        q[i] = j < nq ? qs[j] : zero;
        k[i] = j < nk ? ks[j] : zero;
        v[i] = j < nv ? vs[j] : zero;
    }
#pragma unroll
    for (int i = 0; i < NV; i++) {
        sq += q[i].x * q[i].x + q[i].y * q[i].y + q[i].z * q[i].z + q[i].w * q[i].w;
        sk += k[i].x * k[i].x + k[i].y * k[i].y + k[i].z * k[i].z + k[i].w * k[i].w;
    }
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if ((t & 31u) == 0) { s_part[0][t >> 5] = sq; s_part[1][t >> 5] = sk; }
    __syncthreads();
    sq = sk = 0.f;
#pragma unroll
    for (int i = 0; i < 8; i++) { sq += s_part[0][i]; sk += s_part[1][i]; }
    const float rq = 1.0f / sqrtf(sq / (float)a.q_cols + a.q_eps), rk = 1.0f / sqrtf(sk / (float)a.k_cols + a.k_eps), f = temperature(p, a.coef, a.every);
    auto normed = [](const float4 &x, const float4 &w, float r, float offset, float f) {
        return make_float4(x.x * r * (offset + w.x) * f, x.y * r * (offset + w.y) * f, x.z * r * (offset + w.z) * f, x.w * r * (offset + w.w) * f);
    };
    float *qd = a.q_out + (size_t)row * a.q_cols;
    CT *kd = static_cast<CT *>(a.keys) + (size_t)p * a.k_cols, *vd = static_cast<CT *>(a.values) + (size_t)p * a.v_cols;
#pragma unroll
    for (int i = 0; i < NV; i++) {
        const uint32_t j = t + 256u * i;
        if (j < nq) store4(qd + 4 * j, normed(q[i], __ldg(reinterpret_cast<const float4 *>(a.q_weight) + j), rq, a.q_offset, f));
        if (p >= a.slots) continue;
        if (j < nk) store4(kd + 4 * j, normed(k[i], __ldg(reinterpret_cast<const float4 *>(a.k_weight) + j), rk, a.k_offset, 1.f));
        if (j < nv) store4(vd + 4 * j, v[i]);
    }
}

// CTA = row x {query, key, value}; any width.
template <typename CT>
__global__ void __launch_bounds__(256) attention_inputs_kernel(const __grid_constant__ AttentionInputs a)
{
    constexpr int HOLD = 16;
    __shared__ float s_part[8];
    const uint32_t t = threadIdx.x, row = blockIdx.x, part = blockIdx.y;
    const uint32_t cols = part == 0 ? a.q_cols : part == 1 ? a.k_cols : a.v_cols;
    const float *src = (part == 0 ? a.q : part == 1 ? a.k : a.v) + (size_t)row * cols, *weight = part == 0 ? a.q_weight : a.k_weight;
    pdl_launch_dependents();
    float w[HOLD], v[HOLD];
#pragma unroll
    for (int i = 0; i < HOLD; i++) w[i] = part < 2 && t + 256u * i < cols ? __ldg(weight + t + 256u * i) : 0.f;
    pdl_wait();
    const uint32_t p = a.pos[0] + row;
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < HOLD; i++) {
        v[i] = t + 256u * i < cols ? src[t + 256u * i] : 0.f;
        ss = fmaf(v[i], v[i], ss);
    }
    if (part == 2) {
        if (p >= a.slots) return;
        CT *dst = static_cast<CT *>(a.values) + (size_t)p * cols;
#pragma unroll
        for (int i = 0; i < HOLD; i++)
            if (t + 256u * i < cols) dst[t + 256u * i] = from_f32<CT>(v[i]);
        for (uint32_t j = t + 256u * HOLD; j < cols; j += 256) dst[j] = from_f32<CT>(src[j]);
        return;
    }
    for (uint32_t j = t + 256u * HOLD; j < cols; j += 256) ss = fmaf(src[j], src[j], ss);
    ss = warp_sum(ss);
    if ((t & 31u) == 0) s_part[t >> 5] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; i++) ss += s_part[i];
    const float r = 1.0f / sqrtf(ss / (float)cols + (part == 0 ? a.q_eps : a.k_eps)), offset = part == 0 ? a.q_offset : a.k_offset;
    if (part == 0) {
        const float f = temperature(p, a.coef, a.every);
        float *dst = a.q_out + (size_t)row * cols;
#pragma unroll
        for (int i = 0; i < HOLD; i++)
            if (t + 256u * i < cols) dst[t + 256u * i] = v[i] * r * (offset + w[i]) * f;
        for (uint32_t j = t + 256u * HOLD; j < cols; j += 256) dst[j] = src[j] * r * (offset + weight[j]) * f;
    } else if (p < a.slots) {
        CT *dst = static_cast<CT *>(a.keys) + (size_t)p * cols;
#pragma unroll
        for (int i = 0; i < HOLD; i++)
            if (t + 256u * i < cols) dst[t + 256u * i] = from_f32<CT>(v[i] * r * (offset + w[i]));
        for (uint32_t j = t + 256u * HOLD; j < cols; j += 256) dst[j] = from_f32<CT>(src[j] * r * (offset + weight[j]));
    }
}

// ---------------------------------------------------------------- slices
// Slices share out the keys that the CTA's last row sees, in whole tiles; a slice may be empty.
struct Slice {
    uint32_t k0, k1;                       // keys [k0, k1)
};
__device__ __forceinline__ Slice key_slice(uint32_t total, uint32_t split, uint32_t splits, uint32_t tile)
{
    const uint32_t per = ((total + splits - 1) / splits + tile - 1) / tile * tile, k0 = min(split * per, total);
    return Slice{k0, min(k0 + per, total)};
}
// Pair i of a key / value head: row i / ratio, query head kv_head * ratio + i % ratio.  Partials of a (row, head)
// lie at part = (row * heads + head) * splits + split: `vdim` unnormalised sums, and (maximum, sum of weights).
__device__ __forceinline__ size_t pair_part(const Attention &a, uint32_t kv_head, uint32_t pair, uint32_t split, uint32_t splits)
{
    const uint32_t ratio = a.heads / a.kv_heads, row = pair / ratio, head = kv_head * ratio + pair - row * ratio;
    return ((size_t)row * a.heads + head) * splits + split;
}

// ---------------------------------------------------------------- few rows, any size
constexpr uint32_t kPairs = 8, kTile = 32, kCols = 256;

template <typename CT> __host__ __device__ inline uint32_t row_pitch(uint32_t width)       // an odd number of 16-byte pieces
{
    constexpr uint32_t per = 16 / sizeof(CT);
    return ((width + per - 1) / per | 1u) * per;
}
template <typename CT> size_t general_smem(uint32_t dim, uint32_t vdim)
{
    return (size_t)kPairs * row_pitch<CT>(dim) * sizeof(float) + (size_t)kTile * (row_pitch<CT>(dim) + row_pitch<CT>(std::min(vdim, kCols))) * sizeof(CT);
}

__device__ __forceinline__ void unpack_piece(const float *p, float (&f)[4])
{
    const float4 v = *reinterpret_cast<const float4 *>(p);
    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
}
__device__ __forceinline__ void unpack_piece(const __half *p, float (&f)[8])
{
    const uint4 v = *reinterpret_cast<const uint4 *>(p);
    const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const float2 x = __half22float2(*reinterpret_cast<const __half2 *>(&w[i]));
        f[2 * i] = x.x; f[2 * i + 1] = x.y;
    }
}

template <typename CT>
__global__ void __launch_bounds__(256) attention_kernel(const __grid_constant__ Attention a, float *po, float *ml)
{
    constexpr uint32_t PER = 16 / sizeof(CT);
    extern __shared__ __align__(16) float smem[];
    const uint32_t t = threadIdx.x, lane = t & 31u, warp = t >> 5, vblocks = (a.vdim + kCols - 1) / kCols, kv_head = blockIdx.x / vblocks;
    const uint32_t v0 = blockIdx.x % vblocks * kCols, vcols = min(a.vdim - v0, kCols), split = blockIdx.y, splits = gridDim.y, p0 = blockIdx.z * kPairs;
    const uint32_t ratio = a.heads / a.kv_heads, pairs = a.rows * ratio, kp = row_pitch<CT>(a.dim), vp = row_pitch<CT>(vcols);
    float *s_q = smem;                                                   // [8][kp]
    CT *s_k = reinterpret_cast<CT *>(smem + kPairs * kp), *s_v = s_k + kTile * kp;
    pdl_launch_dependents();
    for (uint32_t i = t; i < kTile * (kp - a.dim); i += 256) s_k[i / (kp - a.dim) * kp + a.dim + i % (kp - a.dim)] = from_f32<CT>(0.f);
    pdl_wait();
    const uint32_t pos0 = a.pos[0], total = min(pos0 + (min(p0 + kPairs, pairs) - 1) / ratio, a.slots - 1) + 1;
    const Slice sl = key_slice(total, split, splits, kTile);
    const uint32_t pair = p0 + warp;
    const bool live = pair < pairs;
    const size_t part = pair_part(a, kv_head, live ? pair : 0, split, splits);
    if (sl.k0 >= sl.k1) {                                                // uniform over the CTA
        if (live && lane == 0 && v0 == 0) { ml[part * 2] = -INFINITY; ml[part * 2 + 1] = 0.f; }
        return;
    }
    for (uint32_t i = t; i < kPairs * kp; i += 256) {
        const uint32_t pr = p0 + i / kp, d = i % kp, row = pr / ratio;
        s_q[i] = pr < pairs && d < a.dim ? a.q[((size_t)row * a.heads + kv_head * ratio + pr - row * ratio) * a.dim + d] : 0.f;
    }
    const CT *keys = static_cast<const CT *>(a.keys) + (size_t)kv_head * a.dim, *values = static_cast<const CT *>(a.values) + (size_t)kv_head * a.vdim + v0;
    const uint32_t see = live ? pos0 + pair / ratio : 0;                 // last visible key
    const float scale = a.scale * kLog2e;
    float acc[kCols / 32], m = -INFINITY, l = 0.f;
#pragma unroll
    for (int i = 0; i < (int)kCols / 32; i++) acc[i] = 0.f;
    for (uint32_t kt = sl.k0; kt < sl.k1; kt += kTile) {
        __syncthreads();
        for (uint32_t r = warp; r < kTile; r += 8) {
            const bool in = kt + r < sl.k1;
            for (uint32_t j = lane; j < a.dim; j += 32) s_k[r * kp + j] = in ? keys[(size_t)(kt + r) * a.kv_heads * a.dim + j] : from_f32<CT>(0.f);
            for (uint32_t j = lane; j < vcols; j += 32) s_v[r * vp + j] = in ? values[(size_t)(kt + r) * a.kv_heads * a.vdim + j] : from_f32<CT>(0.f);
        }
        __syncthreads();
        float s4[4] = {0.f, 0.f, 0.f, 0.f};
        const CT *kr = s_k + lane * kp;
        const float *q = s_q + warp * kp;
#pragma unroll 4
        for (uint32_t d = 0; d < a.dim; d += PER) {                      // query and key are zero beyond dim
            float kv[PER];
            unpack_piece(kr + d, kv);
#pragma unroll
            for (int j = 0; j < (int)PER; j += 4) {
                const float4 x = *reinterpret_cast<const float4 *>(q + d + j);
                s4[0] = fmaf(kv[j], x.x, s4[0]); s4[1] = fmaf(kv[j + 1], x.y, s4[1]);
                s4[2] = fmaf(kv[j + 2], x.z, s4[2]); s4[3] = fmaf(kv[j + 3], x.w, s4[3]);
            }
        }
        const uint32_t key = kt + lane;
        const float s = live && key < sl.k1 && key <= see ? ((s4[0] + s4[1]) + (s4[2] + s4[3])) * scale : -INFINITY;
        const float m_new = fmaxf(m, warp_max(s)), base = m_new == -INFINITY ? 0.f : m_new;
        const float corr = exp2f(m - base), p = exp2f(s - base);         // nothing seen yet: exp2(-inf) = 0
        l = l * corr + warp_sum(p);
        m = m_new;
#pragma unroll
        for (int i = 0; i < (int)kCols / 32; i++) {
            if (32u * i >= vcols) break;
            float o = acc[i] * corr;
#pragma unroll 8
            for (uint32_t k = 0; k < kTile; k++) {
                const float w = __shfl_sync(0xffffffffu, p, k);
                if (lane + 32u * i < vcols) o = fmaf(w, to_f32(s_v[k * vp + lane + 32u * i]), o);
            }
            acc[i] = o;
        }
    }
    if (!live) return;
    float *dst = po + part * a.vdim + v0;
#pragma unroll
    for (int i = 0; i < (int)kCols / 32; i++)
        if (lane + 32u * i < vcols) dst[lane + 32u * i] = acc[i];
    if (lane == 0 && v0 == 0) { ml[part * 2] = m; ml[part * 2 + 1] = l; }
}

// ---------------------------------------------------------------- few rows on the tensor cores
__device__ __forceinline__ uint32_t smem_addr(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp_async16(uint32_t smem, const void *gmem)
{
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(smem), "l"(gmem) : "memory");
}
__device__ __forceinline__ void ldmatrix4(uint32_t addr, uint32_t (&r)[4])
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldmatrix4_t(uint32_t addr, uint32_t (&r)[4])
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1)
{
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack2(float x, float y)
{
    const __half2 h = __floats2half2_rn(x, y);
    return *reinterpret_cast<const uint32_t *>(&h);
}

constexpr uint32_t kMmaPairs = 16, kMmaWarps = 4, kWarpKeys = 16, kMmaTile = kMmaWarps * kWarpKeys, kMmaStages = 3;
__host__ __device__ inline uint32_t mma_pitch(uint32_t width) { return (width + 15u) / 16u * 16u + 8u; }      // an odd number of 16-byte pieces
size_t mma_smem(uint32_t dim, uint32_t dv) { return ((size_t)kMmaPairs * mma_pitch(dim) + (size_t)kMmaStages * kMmaTile * (mma_pitch(dim) + dv + 8)) * 2; }

// DV: value columns of the CTA.
template <int DV>
__global__ void __launch_bounds__(128) attention_mma_kernel(const __grid_constant__ Attention a, float *po, float *ml)
{
    constexpr uint32_t PV = DV + 8;
    extern __shared__ __align__(16) __half sm[];
    __shared__ float s_m[kMmaWarps][kMmaPairs], s_l[kMmaWarps][kMmaPairs];
    const uint32_t t = threadIdx.x, lane = t & 31u, warp = t >> 5, vblocks = (a.vdim + DV - 1) / DV, kv_head = blockIdx.x / vblocks;
    const uint32_t v0 = blockIdx.x % vblocks * DV, vcols = min(a.vdim - v0, (uint32_t)DV), split = blockIdx.y, splits = gridDim.y, p0 = blockIdx.z * kMmaPairs;
    const uint32_t ratio = a.heads / a.kv_heads, pairs = a.rows * ratio, kp = mma_pitch(a.dim), k16 = (a.dim + 15u) / 16u;
    const uint32_t stage_len = kWarpKeys * (kp + PV);                    // elements of one stage of one warp: 16 keys, 16 values
    __half *s_q = sm, *mine = sm + kMmaPairs * kp + warp * kMmaStages * stage_len;
    const __half zero = __float2half_rn(0.f);
    pdl_launch_dependents();
    // zero padding columns: they meet in products
    const uint32_t kpad = k16 * 16 - a.dim, vpad = DV - vcols;
    for (uint32_t s = 0; s < kMmaStages; s++) {
        __half *sk = mine + s * stage_len, *sv = sk + kWarpKeys * kp;
        for (uint32_t i = lane; i < kWarpKeys * kpad; i += 32) sk[i / kpad * kp + a.dim + i % kpad] = zero;
        for (uint32_t i = lane; i < kWarpKeys * vpad; i += 32) sv[i / vpad * PV + vcols + i % vpad] = zero;
    }
    pdl_wait();
    const uint32_t pos0 = a.pos[0], total = min(pos0 + (min(p0 + kMmaPairs, pairs) - 1) / ratio, a.slots - 1) + 1;
    const Slice sl = key_slice(total, split, splits, kMmaTile);
    if (sl.k0 >= sl.k1) {
        if (v0 == 0 && t < kMmaPairs && p0 + t < pairs) {
            float *dst = ml + pair_part(a, kv_head, p0 + t, split, splits) * 2;
            dst[0] = -INFINITY; dst[1] = 0.f;
        }
        return;
    }
    const __half *keys = static_cast<const __half *>(a.keys) + (size_t)kv_head * a.dim, *values = static_cast<const __half *>(a.values) + (size_t)kv_head * a.vdim + v0;
    const size_t krow = (size_t)a.kv_heads * a.dim, vrow = (size_t)a.kv_heads * a.vdim;
    auto stage = [&](uint32_t it) {                                      // this warp's 16 keys of tile `it`; always one commit
        const uint32_t kt = sl.k0 + it * kMmaTile + warp * kWarpKeys;
        if (kt < sl.k1) {
            const uint32_t kb = smem_addr(mine + it % kMmaStages * stage_len), vb = kb + kWarpKeys * kp * 2;
            for (uint32_t r = lane >> 2; r < kWarpKeys; r += 8) {
                const size_t key = min(kt + r, sl.k1 - 1);               // beyond the last key: a valid row, masked below
                for (uint32_t c = (lane & 3u) * 8; c < a.dim; c += 32) cp_async16(kb + (r * kp + c) * 2, keys + key * krow + c);
                for (uint32_t c = (lane & 3u) * 8; c < vcols; c += 32) cp_async16(vb + (r * PV + c) * 2, values + key * vrow + c);
            }
        }
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };
    const uint32_t tiles = (sl.k1 - sl.k0 + kMmaTile - 1) / kMmaTile;
    stage(0);
    stage(1);
    for (uint32_t i = t; i < kMmaPairs * k16 * 8; i += 128) {            // queries, two elements at a time
        const uint32_t pr = i / (k16 * 8), d = i % (k16 * 8) * 2, pair = p0 + pr, row = pair / ratio;
        float2 q = make_float2(0.f, 0.f);
        if (pair < pairs && d < a.dim) q = *reinterpret_cast<const float2 *>(a.q + ((size_t)row * a.heads + kv_head * ratio + pair - row * ratio) * a.dim + d);
        *reinterpret_cast<__half2 *>(s_q + pr * kp + d) = __halves2half2(from_f32<__half>(q.x), from_f32<__half>(q.y));
    }
    __syncthreads();
    float o[DV / 8][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
    for (int n = 0; n < DV / 8; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) o[n][e] = 0.f;
    const uint32_t see[2] = {pos0 + (p0 + lane / 4) / ratio, pos0 + (p0 + lane / 4 + 8) / ratio};      // last visible keys of this thread's pairs
    const uint32_t a_addr = smem_addr(s_q + ((lane & 7u) + ((lane >> 3) & 1u) * 8) * kp + (lane >> 4) * 8);
    const uint32_t b_off = (((lane & 7u) + (lane >> 4) * 8) * kp + ((lane >> 3) & 1u) * 8) * 2;
    const uint32_t v_off = (kWarpKeys * kp + ((lane & 7u) + ((lane >> 3) & 1u) * 8) * PV + (lane >> 4) * 8) * 2;
    const float scale = a.scale * kLog2e;
    for (uint32_t it = 0; it < tiles; it++) {
        asm volatile("cp.async.wait_group 1;\n" ::: "memory");
        __syncwarp();                                                    // the other lanes' copies too, and all have left the buffer that is filled now
        stage(it + 2);
        const uint32_t kt = sl.k0 + it * kMmaTile + warp * kWarpKeys;
        if (kt >= sl.k1) break;
        const uint32_t base = smem_addr(mine + it % kMmaStages * stage_len);
        float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll 4
        for (uint32_t kk = 0; kk < k16; kk++) {
            uint32_t q[4], b[4];
            ldmatrix4(a_addr + kk * 32, q);
            ldmatrix4(base + b_off + kk * 32, b);
            mma16816(s[0], q, b[0], b[1]);
            mma16816(s[1], q, b[2], b[3]);
        }
#pragma unroll
        for (int h = 0; h < 2; h++) {
            float mx = -INFINITY;
#pragma unroll
            for (int n = 0; n < 2; n++)
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    float &x = s[n][2 * h + e];
                    const uint32_t key = kt + n * 8 + (lane & 3u) * 2 + e;
                    x = key <= see[h] && key < sl.k1 ? x * scale : -INFINITY;
                    mx = fmaxf(mx, x);
                }
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
            const float m_new = fmaxf(m[h], mx), top = m_new == -INFINITY ? 0.f : m_new;
            const float corr = exp2f(m[h] - top);        // nothing seen yet: exp2(-inf) = 0
            m[h] = m_new;
            float sum = 0.f;
#pragma unroll
            for (int n = 0; n < 2; n++)
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    float &x = s[n][2 * h + e];
                    x = exp2f(x - top);
                    sum += x;
                }
            l[h] = l[h] * corr + sum;
#pragma unroll
            for (int n = 0; n < DV / 8; n++) { o[n][2 * h] *= corr; o[n][2 * h + 1] *= corr; }
        }
        const uint32_t w[4] = {pack2(s[0][0], s[0][1]), pack2(s[0][2], s[0][3]), pack2(s[1][0], s[1][1]), pack2(s[1][2], s[1][3])};
#pragma unroll
        for (int n = 0; n < DV / 16; n++) {
            uint32_t b[4];
            ldmatrix4_t(base + v_off + n * 32, b);
            mma16816(o[2 * n], w, b[0], b[1]);
            mma16816(o[2 * n + 1], w, b[2], b[3]);
        }
    }
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    // the warps' softmaxes become one
#pragma unroll
    for (int h = 0; h < 2; h++) {
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 1);
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 2);
        if ((lane & 3u) == 0) { s_m[warp][lane / 4 + 8 * h] = m[h]; s_l[warp][lane / 4 + 8 * h] = l[h]; }
    }
    __syncthreads();
    float *s_o = reinterpret_cast<float *>(sm + kMmaPairs * kp);         // [warps][pairs][DV], over the stages
#pragma unroll
    for (int h = 0; h < 2; h++) {
        const uint32_t pr = lane / 4 + 8 * h;
        float top = s_m[0][pr];
#pragma unroll
        for (uint32_t i = 1; i < kMmaWarps; i++) top = fmaxf(top, s_m[i][pr]);
        const float f = top == -INFINITY ? 0.f : exp2f(m[h] - top);
#pragma unroll
        for (int n = 0; n < DV / 8; n++)
            *reinterpret_cast<float2 *>(s_o + (warp * kMmaPairs + pr) * DV + n * 8 + (lane & 3u) * 2) = make_float2(o[n][2 * h] * f, o[n][2 * h + 1] * f);
    }
    __syncthreads();
    for (uint32_t i = t; i < kMmaPairs * DV; i += 128) {
        const uint32_t pr = i / DV, c = i % DV;
        if (p0 + pr >= pairs) break;
        if (c >= vcols) continue;
        float x = 0.f;
#pragma unroll
        for (uint32_t w = 0; w < kMmaWarps; w++) x += s_o[(w * kMmaPairs + pr) * DV + c];
        po[pair_part(a, kv_head, p0 + pr, split, splits) * a.vdim + v0 + c] = x;
    }
    if (v0 == 0 && t < kMmaPairs && p0 + t < pairs) {
        float top = -INFINITY, sum = 0.f;
#pragma unroll
        for (uint32_t w = 0; w < kMmaWarps; w++) top = fmaxf(top, s_m[w][t]);
#pragma unroll
        for (uint32_t w = 0; w < kMmaWarps; w++) sum += top == -INFINITY ? 0.f : s_l[w][t] * exp2f(s_m[w][t] - top);
        float *dst = ml + pair_part(a, kv_head, p0 + t, split, splits) * 2;
        dst[0] = top; dst[1] = sum;
    }
}

// ---------------------------------------------------------------- merge and gate: CTA = (row, head)
template <typename OT>
__global__ void __launch_bounds__(128) attention_merge_kernel(const float *po, const float *ml, uint32_t splits, uint32_t vdim, const __grid_constant__ HeadGate hg, OT *out)
{
    extern __shared__ float s_w[];                       // slice weights [splits]
    const uint32_t t = threadIdx.x, lane = t & 31u, warp = t >> 5;
    const size_t part = (size_t)blockIdx.x * splits;
    pdl_launch_dependents();
    pdl_wait();
    float m = -INFINITY, l = 0.f;
    for (uint32_t s = lane; s < splits; s += 32) m = fmaxf(m, ml[(part + s) * 2]);
    m = warp_max(m);                                     // a row sees at least its own key: finite
    for (uint32_t s = lane; s < splits; s += 32) {
        const float w = exp2f(ml[(part + s) * 2] - m);
        if (warp == 0) s_w[s] = w;
        l = fmaf(ml[(part + s) * 2 + 1], w, l);
    }
    const float inv = 1.0f / warp_sum(l);
    __syncthreads();
    for (uint32_t v = t; v < vdim; v += 128) {
        const float *src = po + part * vdim + v;
        float x = 0.f;
#pragma unroll 16
        for (uint32_t s = 0; s < splits; s++) {
            const float w = s_w[s];
            x = w != 0.f ? fmaf(src[(size_t)s * vdim], w, x) : x;      // an empty slice has no partial
        }
        x *= inv;
        const size_t at = (size_t)blockIdx.x * vdim + v;
        if (hg.gate) {
            const float g = hg.gate[at], sg = sigmoid_f(g);
            x *= hg.silu ? g * sg : sg;
        }
        out[at] = from_f32<OT>(x);
    }
}

size_t align256(size_t n) { return (n + 255) & ~(size_t)255; }

bool mma_eligible(uint32_t dim, uint32_t vdim, bool half) { return half && dim % 8 == 0 && vdim % 8 == 0 && mma_smem(dim, vdim <= 64 ? 64 : 128) <= 210 * 1024; }

// Slices of the keys: enough CTAs for two per SM, none shorter than a tile of 64 keys.
uint32_t key_splits(uint32_t rows, uint32_t heads, uint32_t kv_heads, uint32_t dim, uint32_t vdim, uint32_t slots, bool half)
{
    const bool mma = mma_eligible(dim, vdim, half);
    const uint32_t per = mma ? kMmaPairs : kPairs, cols = mma ? (vdim <= 64 ? 64u : 128u) : kCols;
    const uint32_t ctas = kv_heads * ((vdim + cols - 1) / cols) * ((rows * (heads / kv_heads) + per - 1) / per);
    return std::max(1u, std::min((296u + ctas - 1) / ctas, (slots + 63) / 64));
}

template <int DV>
int launch_mma(const Attention &a, float *po, float *ml, uint32_t splits, cudaStream_t st)
{
    const size_t smem = mma_smem(a.dim, DV);
    if (int rc = allow_smem(attention_mma_kernel<DV>, smem)) return rc;
    const dim3 grid(a.kv_heads * ((a.vdim + DV - 1) / DV), splits, (a.rows * (a.heads / a.kv_heads) + kMmaPairs - 1) / kMmaPairs);
    return launch(attention_mma_kernel<DV>, grid, dim3(128), smem, st, a, po, ml);
}

template <typename CT>
int launch_general(const Attention &a, float *po, float *ml, uint32_t splits, cudaStream_t st)
{
    const size_t smem = general_smem<CT>(a.dim, a.vdim);
    if (smem > 220 * 1024) return fail(MGQ_ERR_SHAPE, "attention: heads of %u dimensions are too wide", a.dim);
    if (int rc = allow_smem(attention_kernel<CT>, smem)) return rc;
    const dim3 grid(a.kv_heads * ((a.vdim + kCols - 1) / kCols), splits, (a.rows * (a.heads / a.kv_heads) + kPairs - 1) / kPairs);
    return launch(attention_kernel<CT>, grid, dim3(256), smem, st, a, po, ml);
}

}  // namespace

int launch_query_temperature(const float *x, const uint32_t *pos, float *out, uint32_t rows, uint32_t cols, float coef, float every, void *stream)
{
    return launch(query_temperature_kernel, dim3((uint32_t)(((size_t)rows * cols + 255) / 256)), dim3(256), 0, static_cast<cudaStream_t>(stream), x, pos, out, rows, cols, coef, every);
}

int launch_cache_append(const float *x, void *cache, bool half, const uint32_t *pos, uint32_t rows, uint32_t cols, uint32_t slots, void *stream)
{
    const dim3 grid((uint32_t)(((size_t)rows * cols + 255) / 256));
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (half) return launch(cache_append_kernel<__half>, grid, dim3(256), 0, st, x, static_cast<__half *>(cache), pos, rows, cols, slots);
    return launch(cache_append_kernel<float>, grid, dim3(256), 0, st, x, static_cast<float *>(cache), pos, rows, cols, slots);
}

int launch_attention_inputs(const AttentionInputs &a, void *stream)
{
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    const uint32_t widest = std::max(a.q_cols, std::max(a.k_cols, a.v_cols));
    if ((a.q_cols | a.k_cols | a.v_cols) % 4 == 0 && widest <= 4096) {
        if (widest <= 2048)
            return a.half ? launch(attention_inputs_vec_kernel<__half, 2>, dim3(a.rows), dim3(256), 0, st, a) : launch(attention_inputs_vec_kernel<float, 2>, dim3(a.rows), dim3(256), 0, st, a);
        return a.half ? launch(attention_inputs_vec_kernel<__half, 4>, dim3(a.rows), dim3(256), 0, st, a) : launch(attention_inputs_vec_kernel<float, 4>, dim3(a.rows), dim3(256), 0, st, a);
    }
    if (a.half) return launch(attention_inputs_kernel<__half>, dim3(a.rows, 3), dim3(256), 0, st, a);
    return launch(attention_inputs_kernel<float>, dim3(a.rows, 3), dim3(256), 0, st, a);
}

size_t attention_workspace(uint32_t max_rows, uint32_t heads, uint32_t kv_heads, uint32_t dim, uint32_t vdim, uint32_t slots, bool half)
{
    // the number of slices falls as the rows grow, their product need not: take the largest
    const bool prefill = half && dim % 8 == 0 && vdim % 8 == 0 && dim <= 256;
    const uint32_t most = prefill ? std::min(max_rows, kPrefillRows - 1) : max_rows;
    size_t parts = 0;
    for (uint32_t r = 1; r <= most; r++) parts = std::max(parts, (size_t)r * key_splits(r, heads, kv_heads, dim, vdim, slots, half));
    return align256(parts * heads * vdim * 4) + align256(parts * heads * 8);
}

int launch_attention(const Attention &a, void *stream)
{
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (a.rows > a.slots) return fail(MGQ_ERR_SHAPE, "attention: %u rows over a cache of %u", a.rows, a.slots);
    if (attention_prefill_eligible(a)) return launch_attention_prefill(a, stream);
    const uint32_t splits = key_splits(a.rows, a.heads, a.kv_heads, a.dim, a.vdim, a.slots, a.half);
    float *po = static_cast<float *>(a.workspace);
    float *ml = reinterpret_cast<float *>(static_cast<uint8_t *>(a.workspace) + align256((size_t)a.rows * splits * a.heads * a.vdim * 4));
    int rc;
    if (mma_eligible(a.dim, a.vdim, a.half)) rc = a.vdim <= 64 ? launch_mma<64>(a, po, ml, splits, st) : launch_mma<128>(a, po, ml, splits, st);
    else rc = a.half ? launch_general<__half>(a, po, ml, splits, st) : launch_general<float>(a, po, ml, splits, st);
    if (rc) return rc;
    const HeadGate none{};
    const HeadGate &hg = a.gate ? *a.gate : none;
    void *out = a.gate ? a.gate->out : a.o;
    const dim3 grid(a.rows * a.heads);
    if (a.gate && a.gate->out_bf16) return launch(attention_merge_kernel<__nv_bfloat16>, grid, dim3(128), splits * 4, st, po, ml, splits, a.vdim, hg, static_cast<__nv_bfloat16 *>(out));
    return launch(attention_merge_kernel<float>, grid, dim3(128), splits * 4, st, po, ml, splits, a.vdim, hg, static_cast<float *>(out));
}

}  // namespace mgq
