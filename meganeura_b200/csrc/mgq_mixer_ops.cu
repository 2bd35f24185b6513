// Embedding, norms, token shift, recurrences (RWKV-style time mixing, gated linear attention, mLSTM
// matrix memory), per-head output gates and the GLU.  All statistics, gates, decays and recurrent state are f32; only the
// operands of the next projection may be stored as bf16.
//
// The recurrences share one schedule.  A head's state is kept value-major, [value][key], and a
// thread owns RPT keys of a few value columns (8 threads per group of columns), so a token step is
// register arithmetic plus a short shuffle reduction; keys beyond `dim` are zero.
//   scan_kernel  several tokens: CTA = head x a block of value columns (x a segment of a long portion),
//                state in registers, the tokens' vectors staged through a double-buffered cp.async ring.
//   step_kernel  one token: a cluster per head, its CTAs share out the value columns; the decay projection (or
//                the gates), the recurrence, the per-head norm (the CTAs' sums of squares meet through distributed
//                shared memory) and the output gate in one launch, state streamed once.
#include <algorithm>

#include "mgq_mixer.cuh"

namespace mgq {
namespace {

__device__ __forceinline__ float block_sum(float v, float *s_part)
{
    v = warp_sum(v);
    __syncthreads();
    if ((threadIdx.x & 31u) == 0) s_part[threadIdx.x >> 5] = v;
    __syncthreads();
    float total = 0.f;
    for (uint32_t i = 0; i < blockDim.x / 32; i++) total += s_part[i];
    return total;
}

template <typename OT> __device__ __forceinline__ void store4(OT *p, float a, float b, float c, float d);
template <> __device__ __forceinline__ void store4<float>(float *p, float a, float b, float c, float d) { *reinterpret_cast<float4 *>(p) = make_float4(a, b, c, d); }
template <> __device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16 *p, float a, float b, float c, float d)
{
    const __nv_bfloat162 x = __floats2bfloat162_rn(a, b), y = __floats2bfloat162_rn(c, d);
    *reinterpret_cast<uint2 *>(p) = make_uint2(*reinterpret_cast<const uint32_t *>(&x), *reinterpret_cast<const uint32_t *>(&y));
}

// ---------------------------------------------------------------- embedding, rows, element-wise
// Sine and cosine of p * f for f = f.x + f.y: the product's rounding error and the low part of f enter as a small angle.
__device__ __forceinline__ void sincos_product(float p, float2 f, float &s, float &c)
{
    const float hi = p * f.x, lo = fmaf(p, f.y, fmaf(p, f.x, -hi));
    float s0, c0;
    sincosf(hi, &s0, &c0);
    const float h = -0.5f * lo * lo;
    s = fmaf(h, s0, fmaf(lo, c0, s0));
    c = fmaf(h, c0, fmaf(-lo, s0, c0));
}

template <typename T>
__global__ void embedding_scaled_kernel(const __grid_constant__ Embedding a)
{
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    pdl_launch_dependents();
    pdl_wait();
    if (i >= (size_t)a.rows * a.width) return;
    const uint32_t row = (uint32_t)(i / a.width), col = (uint32_t)(i - (size_t)row * a.width);
    float x = to_f32(static_cast<const T *>(a.table)[(size_t)min(a.ids[row], a.vocab - 1u) * a.width + col]) * a.scale;
    if (a.sinusoid) {
        float s, c;
        sincos_product((float)(a.pos[0] + row), a.sinusoid[col / 2], s, c);
        x += col & 1u ? c : s;
    }
    a.out[i] = x;
    if (a.copy) a.copy[i] = __float2bfloat16_rn(x);
}

// 8 elements per thread (width % 8 == 0)
template <typename T>
__global__ void embedding_vec_kernel(const __grid_constant__ Embedding a)
{
    const size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * 8;
    pdl_launch_dependents();
    pdl_wait();
    if (i >= (size_t)a.rows * a.width) return;
    const uint32_t row = (uint32_t)(i / a.width), col = (uint32_t)(i - (size_t)row * a.width);
    float f[8];
    load8(static_cast<const T *>(a.table) + (size_t)min(a.ids[row], a.vocab - 1u) * a.width + col, f);
#pragma unroll
    for (int j = 0; j < 8; j++) f[j] *= a.scale;
    if (a.sinusoid) {
        const float p = (float)(a.pos[0] + row);
#pragma unroll
        for (int j = 0; j < 8; j += 2) {
            float s, c;
            sincos_product(p, a.sinusoid[(col + j) / 2], s, c);
            f[j] += s;
            f[j + 1] += c;
        }
    }
    store4<float>(a.out + i, f[0], f[1], f[2], f[3]);
    store4<float>(a.out + i + 4, f[4], f[5], f[6], f[7]);
    if (a.copy) {
        store4<__nv_bfloat16>(a.copy + i, f[0], f[1], f[2], f[3]);
        store4<__nv_bfloat16>(a.copy + i + 4, f[4], f[5], f[6], f[7]);
    }
}

__global__ void pick_rows_kernel(const float *x, const uint32_t *index, float *out, uint32_t rows, uint32_t src_rows, uint32_t cols)
{
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    pdl_launch_dependents();
    pdl_wait();
    if (i >= (size_t)rows * cols) return;
    const uint32_t row = (uint32_t)(i / cols);
    out[i] = x[(size_t)min(index[row], src_rows - 1u) * cols + (i - (size_t)row * cols)];
}

__global__ void bias_add_kernel(const float *x, const float *bias, float *out, size_t len, uint32_t cols)
{
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    pdl_launch_dependents();
    pdl_wait();
    if (i < len) out[i] = x[i] + bias[i % cols];
}

template <typename OT>
__global__ void glu_kernel(const float *gate, const float *up, OT *out, size_t len, Glu act)
{
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    pdl_launch_dependents();
    pdl_wait();
    if (i < len) out[i] = from_f32<OT>(glu_f(gate[i], up[i], act));
}

__global__ void cast_kernel(const float *x, __nv_bfloat16 *out, size_t len)
{
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    pdl_launch_dependents();
    pdl_wait();
    if (i < len) out[i] = __float2bfloat16_rn(x[i]);
}

__global__ void scaled_sum_kernel(const float *a, const float *b, float *out, size_t len, float sa, float sb)
{
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    pdl_launch_dependents();
    pdl_wait();
    if (i < len) out[i] = fmaf(sa, a[i], sb * b[i]);
}

// ---------------------------------------------------------------- RMS norm with a weight offset, optional row index
template <typename OT>
__global__ void __launch_bounds__(256) norm_kernel(const float *x, const float *weight, const uint32_t *index, OT *out, uint32_t src_rows,
                                                   uint32_t cols, float eps, float offset)
{
    constexpr int HOLD = 16;                     // values a thread keeps between the two passes
    __shared__ float s_part[8];
    const uint32_t t = threadIdx.x;
    if (cols % 4 == 0 && cols <= 4096) {         // float4 form
        const uint32_t n4 = cols / 4;
        float4 w[4], v[4];
        pdl_launch_dependents();
#pragma unroll
        for (int i = 0; i < 4; i++) w[i] = t + 256u * i < n4 ? __ldg(reinterpret_cast<const float4 *>(weight) + t + 256u * i) : make_float4(0.f, 0.f, 0.f, 0.f);
        pdl_wait();
        const float4 *src = reinterpret_cast<const float4 *>(x + (size_t)(index ? min(index[blockIdx.x], src_rows - 1u) : blockIdx.x) * cols);
        OT *dst = out + (size_t)blockIdx.x * cols;
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < 4; i++) {
            v[i] = t + 256u * i < n4 ? src[t + 256u * i] : make_float4(0.f, 0.f, 0.f, 0.f);
            ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
        }
        const float r = 1.0f / sqrtf(block_sum(ss, s_part) / (float)cols + eps);
#pragma unroll
        for (int i = 0; i < 4; i++)
            if (t + 256u * i < n4)
                store4<OT>(dst + 4 * (t + 256u * i), v[i].x * r * (offset + w[i].x), v[i].y * r * (offset + w[i].y), v[i].z * r * (offset + w[i].z),
                           v[i].w * r * (offset + w[i].w));
        return;
    }
    float w[HOLD], v[HOLD];
    pdl_launch_dependents();
#pragma unroll
    for (int i = 0; i < HOLD; i++) w[i] = t + 256u * i < cols ? offset + __ldg(weight + t + 256u * i) : 0.f;
    pdl_wait();
    const uint32_t row = index ? min(index[blockIdx.x], src_rows - 1u) : blockIdx.x;
    const float *src = x + (size_t)row * cols;
    OT *dst = out + (size_t)blockIdx.x * cols;
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < HOLD; i++) {
        v[i] = t + 256u * i < cols ? src[t + 256u * i] : 0.f;
        ss = fmaf(v[i], v[i], ss);
    }
    for (uint32_t j = t + 256u * HOLD; j < cols; j += 256) ss = fmaf(src[j], src[j], ss);
    const float r = 1.0f / sqrtf(block_sum(ss, s_part) / (float)cols + eps);
#pragma unroll
    for (int i = 0; i < HOLD; i++)
        if (t + 256u * i < cols) dst[t + 256u * i] = from_f32<OT>(v[i] * r * w[i]);
    for (uint32_t j = t + 256u * HOLD; j < cols; j += 256) dst[j] = from_f32<OT>(src[j] * r * (offset + weight[j]));
}

// ---------------------------------------------------------------- norm behind a sublayer, added to the residual
// V elements per access.  NV accesses of a row per thread stay in registers; a wider row is summed and read again.
template <int V, int NV>
__global__ void __launch_bounds__(256) residual_norm_kernel(const __grid_constant__ ResidualNorm p)
{
    __shared__ float s_part[8];
    const uint32_t t = threadIdx.x, n = p.cols / V;
    const size_t base = (size_t)blockIdx.x * p.cols;
    auto load = [&](const float *src, uint32_t j, float (&x)[V]) {
        if (V == 4) {
            const float4 f = *reinterpret_cast<const float4 *>(src + 4 * j);
            x[0] = f.x; x[V / 4] = f.y; x[V / 2] = f.z; x[V - 1] = f.w;
        } else {
            x[0] = src[j];
        }
    };
    auto value = [&](uint32_t j, float (&y)[V]) {
        load(p.a + base, j, y);
#pragma unroll
        for (int e = 0; e < V; e++) y[e] *= p.sa;
        if (!p.b) return;
        float z[V];
        load(p.b + base, j, z);
#pragma unroll
        for (int e = 0; e < V; e++) y[e] = fmaf(p.sb, z[e], y[e]);
    };
    float w[NV][V], y[NV][V], x[NV][V];
    pdl_launch_dependents();
#pragma unroll
    for (int i = 0; i < NV; i++)
        if (t + 256u * i < n) load(p.weight, t + 256u * i, w[i]);
    pdl_wait();
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; i++) {
        if (t + 256u * i >= n) break;
        value(t + 256u * i, y[i]);
        load(p.addend + base, t + 256u * i, x[i]);
    }
#pragma unroll
    for (int i = 0; i < NV; i++) {
        if (t + 256u * i >= n) break;
#pragma unroll
        for (int e = 0; e < V; e++) ss = fmaf(y[i][e], y[i][e], ss);
    }
    for (uint32_t j = t + 256u * NV; j < n; j += 256) {
        float z[V];
        value(j, z);
#pragma unroll
        for (int e = 0; e < V; e++) ss = fmaf(z[e], z[e], ss);
    }
    const float r = 1.0f / sqrtf(block_sum(ss, s_part) / (float)p.cols + p.eps);
    auto put = [&](uint32_t j, const float (&yy)[V], const float (&ww)[V], const float (&xx)[V]) {
        float o[V];
#pragma unroll
        for (int e = 0; e < V; e++) o[e] = fmaf(yy[e] * r, p.offset + ww[e], xx[e]);
        if (V == 4) {
            store4<float>(p.out + base + 4 * j, o[0], o[V / 4], o[V / 2], o[V - 1]);
            if (p.copy) store4<__nv_bfloat16>(p.copy + base + 4 * j, o[0], o[V / 4], o[V / 2], o[V - 1]);
        } else {
            p.out[base + j] = o[0];
            if (p.copy) p.copy[base + j] = __float2bfloat16_rn(o[0]);
        }
    };
#pragma unroll
    for (int i = 0; i < NV; i++)
        if (t + 256u * i < n) put(t + 256u * i, y[i], w[i], x[i]);
    for (uint32_t j = t + 256u * NV; j < n; j += 256) {
        float yy[V], ww[V], xx[V];
        value(j, yy);
        load(p.weight, j, ww);
        load(p.addend + base, j, xx);
        put(j, yy, ww, xx);
    }
}

// ---------------------------------------------------------------- token shift (with the norm in front of it)
template <typename OT>
__global__ void __launch_bounds__(256) token_shift_kernel(const __grid_constant__ TokenShift a)
{
    __shared__ float s_part[8];
    const uint32_t t = threadIdx.x, row = blockIdx.x, width = a.width;
    pdl_launch_dependents();
    pdl_wait();
    const float *cur = a.x + (size_t)row * width, *before = row ? cur - width : a.state;
    float r_cur = 1.f, r_before = 1.f;
    if (a.norm_weight) {
        float s0 = 0.f, s1 = 0.f;
        for (uint32_t j = t; j < width; j += 256) {
            s0 = fmaf(cur[j], cur[j], s0);
            if (row) s1 = fmaf(before[j], before[j], s1);
        }
        r_cur = 1.0f / sqrtf(block_sum(s0, s_part) / (float)width + a.eps);
        if (row) r_before = 1.0f / sqrtf(block_sum(s1, s_part) / (float)width + a.eps);
    }
    const bool last = row + 1 == a.rows;
    OT *out = static_cast<OT *>(a.out) + (size_t)row * width;
    for (uint32_t j = t; j < width; j += 256) {
        const float g = a.norm_weight ? a.offset + a.norm_weight[j] : 1.f;
        const float h = a.norm_weight ? cur[j] * r_cur * g : cur[j];
        const float hp = row && a.norm_weight ? before[j] * r_before * g : before[j];        // the state already holds a normed h
        for (uint32_t s = 0; s < a.slots; s++) out[s * a.slot_stride + j] = from_f32<OT>(fmaf(hp - h, a.mu[s][j], h));
        if (last) a.state[width + j] = h;
    }
}

// Vector form: NV float4 of a row per thread, RB consecutive rows per CTA (the previous row stays in
// registers).  A single row is spread over gridDim.y CTAs, each of which sums the whole row and writes
// one group of 1024 channels.
template <typename OT, int NV>
__global__ void __launch_bounds__(256) token_shift_vec_kernel(const __grid_constant__ TokenShift a, uint32_t rows_per_cta)
{
    __shared__ float s_part[8];
    const uint32_t t = threadIdx.x, width = a.width, n4 = width / 4, row0 = blockIdx.x * rows_per_cta, row1 = min(row0 + rows_per_cta, a.rows);
    const bool sliced = gridDim.y > 1;
    float4 g[NV];
    pdl_launch_dependents();
#pragma unroll
    for (int i = 0; i < NV; i++) {
        const uint32_t j = t + 256u * i;
        g[i] = make_float4(1.f, 1.f, 1.f, 1.f);
        if (a.norm_weight && j < n4) {
            const float4 w = __ldg(reinterpret_cast<const float4 *>(a.norm_weight) + j);
            g[i] = make_float4(a.offset + w.x, a.offset + w.y, a.offset + w.z, a.offset + w.w);
        }
        if (sliced && (uint32_t)i == blockIdx.y && j < n4)
            for (uint32_t s = 0; s < a.slots; s++) asm volatile("prefetch.global.L1 [%0];" ::"l"(a.mu[s] + 4 * j));
    }
    pdl_wait();
    auto load_h = [&](uint32_t row, float4 (&h)[NV]) {
        const float4 *src = reinterpret_cast<const float4 *>(a.x + (size_t)row * width);
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < NV; i++) {
            h[i] = t + 256u * i < n4 ? src[t + 256u * i] : make_float4(0.f, 0.f, 0.f, 0.f);
            ss += h[i].x * h[i].x + h[i].y * h[i].y + h[i].z * h[i].z + h[i].w * h[i].w;
        }
        if (!a.norm_weight) return;
        const float r = 1.0f / sqrtf(block_sum(ss, s_part) / (float)width + a.eps);
#pragma unroll
        for (int i = 0; i < NV; i++) { h[i].x *= r * g[i].x; h[i].y *= r * g[i].y; h[i].z *= r * g[i].z; h[i].w *= r * g[i].w; }
    };
    float4 prev[NV], h[NV];
    if (row0) {
        load_h(row0 - 1, prev);
    } else {
#pragma unroll
        for (int i = 0; i < NV; i++) prev[i] = t + 256u * i < n4 ? reinterpret_cast<const float4 *>(a.state)[t + 256u * i] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    for (uint32_t row = row0; row < row1; row++) {
        load_h(row, h);
        OT *out = static_cast<OT *>(a.out) + (size_t)row * width;
#pragma unroll
        for (int i = 0; i < NV; i++) {
            const uint32_t j = t + 256u * i;
            if (j >= n4 || (sliced && (uint32_t)i != blockIdx.y)) continue;
            const float4 d = make_float4(prev[i].x - h[i].x, prev[i].y - h[i].y, prev[i].z - h[i].z, prev[i].w - h[i].w);
            for (uint32_t s = 0; s < a.slots; s++) {
                const float4 m = *(reinterpret_cast<const float4 *>(a.mu[s]) + j);
                store4<OT>(out + s * a.slot_stride + 4 * j, fmaf(d.x, m.x, h[i].x), fmaf(d.y, m.y, h[i].y), fmaf(d.z, m.z, h[i].z), fmaf(d.w, m.w, h[i].w));
            }
            if (row + 1 == a.rows) reinterpret_cast<float4 *>(a.state + width)[j] = h[i];
        }
#pragma unroll
        for (int i = 0; i < NV; i++) prev[i] = h[i];
    }
}

// ---------------------------------------------------------------- per-head norm and gate: one warp per (row, head)
template <typename OT>
__global__ void __launch_bounds__(256) head_gate_kernel(const float *o, const __grid_constant__ HeadGate hg, uint32_t total, uint32_t heads, uint32_t dim)
{
    constexpr int HOLD = 8;
    const uint32_t lane = threadIdx.x & 31u, unit = blockIdx.x * 8u + (threadIdx.x >> 5);
    pdl_launch_dependents();
    pdl_wait();
    if (unit >= total) return;
    const size_t base = (size_t)unit * dim;
    const uint32_t wbase = hg.shared ? 0 : (unit % heads) * dim;
    float v[HOLD], ss = 0.f, r = 1.f;
#pragma unroll
    for (int i = 0; i < HOLD; i++) {
        v[i] = lane + 32u * i < dim ? o[base + lane + 32u * i] : 0.f;
        ss = fmaf(v[i], v[i], ss);
    }
    for (uint32_t j = lane + 32u * HOLD; j < dim; j += 32) ss = fmaf(o[base + j], o[base + j], ss);
    if (hg.weight) r = 1.0f / sqrtf(warp_sum(ss) / (float)dim + hg.eps);
    OT *out = static_cast<OT *>(hg.out);
    auto put = [&](uint32_t j, float val) {
        const float g = hg.gate[base + j], s = sigmoid_f(g);
        out[base + j] = from_f32<OT>(val * r * (hg.weight ? hg.weight[wbase + j] : 1.f) * (hg.silu ? g * s : s));
    };
#pragma unroll
    for (int i = 0; i < HOLD; i++)
        if (lane + 32u * i < dim) put(lane + 32u * i, v[i]);
    for (uint32_t j = lane + 32u * HOLD; j < dim; j += 32) put(j, o[base + j]);
}

// G lanes per (row, head), KV float4 per lane: dim <= 4 * G * KV, dim % 4 == 0.
template <typename OT, int G, int KV>
__global__ void __launch_bounds__(256) head_gate_vec_kernel(const float *o, const __grid_constant__ HeadGate hg, uint32_t total, uint32_t heads, uint32_t dim)
{
    const uint32_t unit = (blockIdx.x * 256u + threadIdx.x) / G, lane = threadIdx.x % G, n4 = dim / 4;
    pdl_launch_dependents();
    pdl_wait();
    const bool live = unit < total;                      // no early return: the lanes of a warp reduce together
    const size_t base = (size_t)(live ? unit : 0) * dim;
    const uint32_t wbase = hg.shared || !live ? 0 : unit % heads * dim;
    float4 v[KV], g[KV];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < KV; i++) {
        const uint32_t j = lane + G * i;
        v[i] = g[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (j < n4) {
            v[i] = *(reinterpret_cast<const float4 *>(o + base) + j);
            g[i] = *(reinterpret_cast<const float4 *>(hg.gate + base) + j);
        }
        ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
    float r = 1.f;
    if (hg.weight) {
#pragma unroll
        for (int off = G / 2; off > 0; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
        r = 1.0f / sqrtf(ss / (float)dim + hg.eps);
    }
    if (!live) return;
    OT *out = static_cast<OT *>(hg.out) + base;
#pragma unroll
    for (int i = 0; i < KV; i++) {
        const uint32_t j = lane + G * i;
        if (j >= n4) break;
        float4 w = make_float4(1.f, 1.f, 1.f, 1.f);
        if (hg.weight) w = *(reinterpret_cast<const float4 *>(hg.weight + wbase) + j);
        auto act = [&](float x) { const float sg = sigmoid_f(x); return hg.silu ? x * sg : sg; };
        store4<OT>(out + 4 * j, v[i].x * r * w.x * act(g[i].x), v[i].y * r * w.y * act(g[i].y), v[i].z * r * w.z * act(g[i].z), v[i].w * r * w.w * act(g[i].w));
    }
}

// ---------------------------------------------------------------- decays, 64 rows x 64 channels per CTA
constexpr uint32_t kDecayTile = 64, kDecayK = 16;
__global__ void __launch_bounds__(256) decay_kernel(const __grid_constant__ Decay a)
{
    __shared__ float s_low[kDecayK][kDecayTile + 4], s_w[kDecayK][kDecayTile + 4];
    const uint32_t t = threadIdx.x, tx = t & 15u, ty = t >> 4, ch0 = blockIdx.x * kDecayTile, row0 = blockIdx.y * kDecayTile, channels = a.channels;
    const __nv_bfloat16 *w = static_cast<const __nv_bfloat16 *>(a.w2);
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) acc[i][j] = 0.f;
    pdl_launch_dependents();
    pdl_wait();
    for (uint32_t k0 = 0; k0 < a.rank; k0 += kDecayK) {
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const uint32_t e = t + 256u * i, r = e / kDecayK, k = e % kDecayK;
            const bool in = k0 + k < a.rank;
            s_low[k][r] = in && row0 + r < a.rows ? decay_input(a.low[(size_t)(row0 + r) * a.rank + k0 + k], a.inv_tau) : 0.f;
            s_w[k][r] = in && ch0 + r < channels ? __bfloat162float(w[(size_t)(ch0 + r) * a.rank + k0 + k]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < (int)kDecayK; k++) {
            const float4 x = *reinterpret_cast<const float4 *>(&s_low[k][ty * 4]), y = *reinterpret_cast<const float4 *>(&s_w[k][tx * 4]);
            const float xr[4] = {x.x, x.y, x.z, x.w}, yr[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(xr[i], yr[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const uint32_t row = row0 + ty * 4 + i;
        if (row >= a.rows) break;
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const uint32_t ch = ch0 + tx * 4 + j;
            if (ch < channels) a.out[(size_t)row * channels + ch] = decay_value(acc[i][j] + a.w0[ch], a.inv_tau);
        }
    }
}

// ---------------------------------------------------------------- recurrences
__device__ __forceinline__ void cp_async4(void *smem, const void *gmem)
{
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"((unsigned)__cvta_generic_to_shared(smem)), "l"(gmem) : "memory");
}
__device__ __forceinline__ void cp_async16(void *smem, const void *gmem)
{
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((unsigned)__cvta_generic_to_shared(smem)), "l"(gmem) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N) : "memory"); }

enum { kWkv = 0, kMlstm = 1, kGla = 2 };

struct Scan {
    const float *q, *k, *v, *w;          // wkv, gla: with a decay per key channel;  mlstm: w unused
    const float *u;                      // wkv bonus [heads, dim]
    const float *gi, *gf;                // mlstm gate pre-activations [rows, heads]
    float *o, *state, *shift_state;
    float *segments;                     // scratch: end states of the segments (several segments only)
    uint32_t rows, heads, dim, vdim, shift_width;
    uint32_t seg_len, seg_count, phase;  // see scan_kernel
    float cap, qscale;
};

__host__ __device__ inline uint32_t pad4(uint32_t d) { return (d + 3u) & ~3u; }
template <int RPT> __host__ __device__ constexpr int chunk_tokens() { return RPT <= 8 ? 32 : RPT == 16 ? 16 : 8; }
// Value columns per thread and per CTA (128 threads, 8 per group of columns): as many as registers hold, since every
// column reuses the key vectors read from shared memory.
template <int RPT> __host__ __device__ constexpr int thread_cols() { return RPT <= 16 ? 4 : 2; }
__host__ __device__ inline uint32_t block_cols(uint32_t dim) { return dim <= 128 ? 64u : 32u; }

// One token of C value columns for the RPT keys this thread owns; OUT: out / den receive its share of the
// dot products.  n: mlstm normalizer; without OUT a thread with channel decays multiplies them into it instead.
template <int MODE, int RPT, int C, bool OUT>
__device__ __forceinline__ void token_update(const float *q, const float *k, const float *w, const float (&u)[RPT], const float (&v_in)[C], float a, float b,
                                             float (&S)[C][RPT], float (&n)[RPT], float (&out)[C], float &den)
{
    float v[C], d = 0.f;
#pragma unroll
    for (int c = 0; c < C; c++) {
        v[c] = MODE == kMlstm ? v_in[c] * b : v_in[c];
        out[c] = 0.f;
    }
#pragma unroll
    for (int i = 0; i < RPT; i += 4) {
        const float4 k4 = *reinterpret_cast<const float4 *>(k + i * 8);
        const float kv[4] = {k4.x, k4.y, k4.z, k4.w};
        float qv[4] = {0.f, 0.f, 0.f, 0.f}, wv[4] = {0.f, 0.f, 0.f, 0.f};
        if (OUT) {
            const float4 q4 = *reinterpret_cast<const float4 *>(q + i * 8);
            qv[0] = q4.x; qv[1] = q4.y; qv[2] = q4.z; qv[3] = q4.w;
        }
        if (MODE != kMlstm) {
            const float4 w4 = *reinterpret_cast<const float4 *>(w + i * 8);
            wv[0] = w4.x; wv[1] = w4.y; wv[2] = w4.z; wv[3] = w4.w;
        }
#pragma unroll
        for (int j = 0; j < 4; j++) {
            if (MODE != kMlstm) {
                if (!OUT) n[i + j] *= wv[j];
#pragma unroll
                for (int c = 0; c < C; c++) {
                    const float x = kv[j] * v[c];
                    if (OUT && MODE == kWkv) out[c] = fmaf(qv[j], fmaf(u[i + j], x, S[c][i + j]), out[c]);
                    S[c][i + j] = fmaf(wv[j], S[c][i + j], x);
                    if (OUT && MODE == kGla) out[c] = fmaf(qv[j], S[c][i + j], out[c]);
                }
            } else {
                n[i + j] = fmaf(kv[j], b, a * n[i + j]);
                if (OUT) d = fmaf(qv[j], n[i + j], d);
#pragma unroll
                for (int c = 0; c < C; c++) {
                    S[c][i + j] = fmaf(kv[j], v[c], a * S[c][i + j]);
                    if (OUT) out[c] = fmaf(qv[j], S[c][i + j], out[c]);
                }
            }
        }
    }
    den = d;
}

__device__ __forceinline__ float sum8(float x)
{
#pragma unroll
    for (int off = 4; off > 0; off >>= 1) x += __shfl_xor_sync(0xffffffffu, x, off);
    return x;
}

// Sums x[t] over the 8 threads of a column for 8 tokens at once: every exchange halves the tokens a
// thread is responsible for; thread ks ends up with the total of token ks.
__device__ __forceinline__ float reduce8(const float (&x)[8], uint32_t ks)
{
    float y[4], z[2];
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const bool up = ks & 4u;
        y[i] = (up ? x[i + 4] : x[i]) + __shfl_xor_sync(0xffffffffu, up ? x[i] : x[i + 4], 4);
    }
#pragma unroll
    for (int i = 0; i < 2; i++) {
        const bool up = ks & 2u;
        z[i] = (up ? y[i + 2] : y[i]) + __shfl_xor_sync(0xffffffffu, up ? y[i] : y[i + 2], 2);
    }
    const bool up = ks & 1u;
    return (up ? z[1] : z[0]) + __shfl_xor_sync(0xffffffffu, up ? z[0] : z[1], 1);
}

__device__ __forceinline__ float mlstm_out(float out, float den, float qscale, float floor_)
{
    return out * qscale / (fmaxf(fabsf(den * qscale), floor_) + 1e-6f);
}

// Keys owned by thread ks of a column: (i * 8 + ks) * 4 + j for i < RPT / 4, j < 4.
template <int RPT>
__device__ __forceinline__ void load_keys(const float *row, uint32_t ks, uint32_t kp, float (&x)[RPT])
{
#pragma unroll
    for (int i = 0; i < RPT; i += 4) {
        const uint32_t at = (i * 2u + ks) * 4u;              // (i / 4 * 8 + ks) * 4
        const float4 v = at < kp ? *reinterpret_cast<const float4 *>(row + at) : make_float4(0.f, 0.f, 0.f, 0.f);
        x[i] = v.x; x[i + 1] = v.y; x[i + 2] = v.z; x[i + 3] = v.w;
    }
}
template <int RPT>
__device__ __forceinline__ void store_keys(float *row, uint32_t ks, uint32_t kp, const float (&x)[RPT])
{
#pragma unroll
    for (int i = 0; i < RPT; i += 4) {
        const uint32_t at = (i * 2u + ks) * 4u;
        if (at < kp) *reinterpret_cast<float4 *>(row + at) = make_float4(x[i], x[i + 1], x[i + 2], x[i + 3]);
    }
}

constexpr uint32_t kScanThreads = 128;

// A state block: [heads][vdim][pad4(dim)], then per head and block of value columns [pad4(dim)] plus 4
// scalars.  In an mlstm state those hold n and m, one copy per block (every CTA of a head advances its own,
// so no CTA reads what another one writes); in a segment's end state also the decay product (per key in
// place of n: channel decays) or the sum of log forget gates (mlstm: scalar 1).
__host__ __device__ inline uint32_t value_blocks(uint32_t dim, uint32_t vdim) { return (vdim + block_cols(dim) - 1) / block_cols(dim); }
__host__ __device__ inline size_t block_elements(uint32_t heads, uint32_t dim, uint32_t vdim)
{
    return (size_t)heads * vdim * pad4(dim) + (size_t)heads * value_blocks(dim, vdim) * (pad4(dim) + 4u);
}
__device__ __forceinline__ float *normalizer(const Scan &p, float *base, uint32_t head, uint32_t block)
{
    const uint32_t kp = pad4(p.dim);
    return base + (size_t)p.heads * p.vdim * kp + (size_t)(head * value_blocks(p.dim, p.vdim) + block) * (kp + 4u);
}

// One launch (phase 0) runs all tokens from the state.  A long portion is cut into segments of seg_len
// tokens and takes two launches of seg_count - 1 segments each: phase 1 runs segment 0 from the state,
// with outputs, and the middle segments from nothing, for their end states only; phase 2 starts segments
// 1.. from the end states before them, put together in order.  Decays are only ever multiplied, and
// mlstm end states carry their own maximum, so nothing can overflow.
template <int MODE, int RPT>
__global__ void __launch_bounds__(kScanThreads, 2) scan_kernel(const __grid_constant__ Scan p)
{
    constexpr int TC = chunk_tokens<RPT>(), KS = RPT * 8, NA = MODE != kMlstm ? 3 : 2, C = thread_cols<RPT>(), COLS = 16 * C;
    extern __shared__ __align__(16) float smem[];
    // per buffer: NA x [TC][KS] key vectors, [TC][COLS] values
    constexpr int kBuf = NA * TC * KS + TC * COLS;
    __shared__ float s_gate[2][3][32];                   // mlstm: keep, write, exp(-m) per token of a chunk
    __shared__ float s_end[2];                           // mlstm: m and the sum of log forget gates at the end
    const uint32_t t = threadIdx.x, head = blockIdx.x, block = blockIdx.y, ks = t & 7u, vc = t / 8 * C, col = block * COLS + vc;
    const uint32_t dim = p.dim, vdim = p.vdim, kp = pad4(dim), kpitch = p.heads * dim, vpitch = p.heads * vdim;
    const uint32_t seg = p.phase == 2 ? blockIdx.z + 1 : blockIdx.z, row0 = seg * p.seg_len, rows = min(p.seg_len, p.rows - row0);
    const bool outputs = p.phase != 1 || seg == 0, from_state = seg == 0;
    const uint32_t chunks = (rows + TC - 1) / TC;
    for (uint32_t i = t; i < 2u * kBuf; i += kScanThreads) smem[i] = 0.f;          // keys beyond dim stay zero
    float S[C][RPT], n[RPT], u[RPT], m = 0.f;
#pragma unroll
    for (int i = 0; i < RPT; i++) {
        const uint32_t key = (i / 4 * 8 + ks) * 4 + i % 4;
        u[i] = MODE == kWkv && key < dim ? __ldg(p.u + head * dim + key) : 0.f;
        n[i] = MODE != kMlstm ? 1.f : 0.f;
#pragma unroll
        for (int c = 0; c < C; c++) S[c][i] = 0.f;
    }
    pdl_launch_dependents();
    pdl_wait();
    __syncthreads();
    const bool vec = dim % 4 == 0 && (reinterpret_cast<uintptr_t>(p.q) | reinterpret_cast<uintptr_t>(p.k) | reinterpret_cast<uintptr_t>(p.w)) % 16 == 0;
    const bool vec_v = vdim % 4 == 0 && COLS % 4 == 0 && (reinterpret_cast<uintptr_t>(p.v) | reinterpret_cast<uintptr_t>(p.o)) % 16 == 0;

    auto stage = [&](uint32_t c, uint32_t buf) {
        float *base = smem + buf * kBuf;
        const uint32_t r0 = row0 + c * TC, cnt = min((uint32_t)TC, rows - c * TC);
#pragma unroll
        for (int arr = 0; arr < NA; arr++) {
            if (arr == 0 && !outputs) continue;
            const float *src = (arr == 0 ? p.q : arr == 1 ? p.k : p.w) + (size_t)r0 * kpitch + head * dim;
            float *dst = base + arr * TC * KS;
            if (vec) {
                for (uint32_t j = (t & 7u) * 4; j < dim; j += 32)
                    for (uint32_t r = t / 8; r < cnt; r += kScanThreads / 8) cp_async16(dst + r * KS + j, src + (size_t)r * kpitch + j);
            } else {
                for (uint32_t j = t & 7u; j < dim; j += 8)
                    for (uint32_t r = t / 8; r < cnt; r += kScanThreads / 8) cp_async4(dst + r * KS + j, src + (size_t)r * kpitch + j);
            }
        }
        float *dv = base + NA * TC * KS;
        const float *sv = p.v + (size_t)r0 * vpitch + head * vdim + block * COLS;
        const uint32_t cols = min((uint32_t)COLS, vdim - block * COLS);
        if (vec_v) {
            for (uint32_t j = (t & 7u) * 4; j < cols; j += 32)
                for (uint32_t r = t / 8; r < cnt; r += kScanThreads / 8) cp_async16(dv + r * COLS + j, sv + (size_t)r * vpitch + j);
        } else {
            for (uint32_t j = t & 7u; j < cols; j += 8)
                for (uint32_t r = t / 8; r < cnt; r += kScanThreads / 8) cp_async4(dv + r * COLS + j, sv + (size_t)r * vpitch + j);
        }
        cp_commit();
    };
    stage(0, 0);

    // the state in front of the segment
    auto load_state = [&](float *base, float (&X)[C][RPT]) {
#pragma unroll
        for (int c = 0; c < C; c++)
            if (col + c < vdim) load_keys<RPT>(base + ((size_t)head * vdim + col + c) * kp, ks, kp, X[c]);
    };
    const size_t stride = block_elements(p.heads, dim, vdim);
    if (from_state) {
        load_state(p.state, S);
        if (MODE == kMlstm) {
            const float *nb = normalizer(p, p.state, head, block);
            load_keys<RPT>(nb, ks, kp, n);
            m = nb[kp];
        }
    } else if (outputs) {
        load_state(p.segments, S);
        if (MODE == kMlstm) {
            const float *nb = normalizer(p, p.segments, head, block);
            load_keys<RPT>(nb, ks, kp, n);
            m = nb[kp];
        }
        for (uint32_t g = 1; g < seg; g++) {
            float *base = p.segments + g * stride;
            const float *nb = normalizer(p, base, head, block);
            float f[RPT];
            load_keys<RPT>(nb, ks, kp, f);
            float keep = 1.f, add = 1.f;
            if (MODE == kMlstm) {
                const float m_new = fmaxf(nb[kp + 1] + m, nb[kp]);
                keep = expf(nb[kp + 1] + m - m_new);
                add = expf(nb[kp] - m_new);
                m = m_new;
#pragma unroll
                for (int i = 0; i < RPT; i++) n[i] = fmaf(add, f[i], keep * n[i]);
            }
#pragma unroll
            for (int c = 0; c < C; c++) {
                if (col + c >= vdim) continue;
                float x[RPT];
                load_keys<RPT>(base + ((size_t)head * vdim + col + c) * kp, ks, kp, x);
#pragma unroll
                for (int i = 0; i < RPT; i++) S[c][i] = MODE != kMlstm ? fmaf(f[i], S[c][i], x[i]) : fmaf(add, x[i], keep * S[c][i]);
            }
        }
    } else if (MODE == kMlstm) {
        m = -INFINITY;
    }
    // mlstm gates of a chunk by one warp: m_t = max(f_t + m_{t-1}, i_t) is a scan of (sum f, max) pairs
    float f_sum = 0.f;
    auto gates = [&](uint32_t c, uint32_t buf) {
        const uint32_t lane = t, row = c * TC + lane, cnt = min((uint32_t)TC, rows - c * TC);
        const bool in = lane < cnt;
        const size_t at = (size_t)(row0 + row) * p.heads + head;
        const float xi = in ? p.gi[at] : 0.f, xf = in ? p.gf[at] : 0.f;
        const float li = p.cap * tanhf(xi / p.cap), lf = in ? log_sigmoid(p.cap * tanhf(xf / p.cap)) : 0.f;
        float F = lf, M = in ? li : -INFINITY;
#pragma unroll
        for (int off = 1; off < 32; off <<= 1) {
            const float Fp = __shfl_up_sync(0xffffffffu, F, off), Mp = __shfl_up_sync(0xffffffffu, M, off);
            if (lane >= (uint32_t)off) { M = fmaxf(M, F + Mp); F += Fp; }
        }
        const float mt = fmaxf(F + m, M);
        float prev = __shfl_up_sync(0xffffffffu, mt, 1);
        if (lane == 0) prev = m;
        s_gate[buf][0][lane] = expf(lf + prev - mt);         // a segment that starts from nothing: exp(-inf) = 0
        s_gate[buf][1][lane] = in ? expf(li - mt) : 0.f;
        s_gate[buf][2][lane] = expf(-mt);
        m = __shfl_sync(0xffffffffu, mt, cnt - 1);
        f_sum += __shfl_sync(0xffffffffu, F, cnt - 1);
    };
    if (MODE == kMlstm && t < 32) gates(0, 0);
    for (uint32_t c = 0; c < chunks; c++) {
        const uint32_t buf = c & 1u;
        if (c + 1 < chunks) { stage(c + 1, buf ^ 1u); cp_wait<1>(); } else { cp_wait<0>(); }
        __syncthreads();
        const float *base = smem + buf * kBuf, *sq = base + ks * 4, *sk = sq + TC * KS, *sw = sk + (NA == 3 ? TC * KS : 0);
        const float *sv = base + NA * TC * KS + vc;
        const uint32_t r0 = row0 + c * TC, cnt = min((uint32_t)TC, rows - c * TC);
        float *dst = p.o + (size_t)r0 * vpitch + head * vdim + col;
        auto values = [&](uint32_t r, float (&v)[C]) {
#pragma unroll
            for (int i = 0; i < C; i += 2) {
                const float2 x = *reinterpret_cast<const float2 *>(sv + r * COLS + i);
                v[i] = x.x; v[i + 1] = x.y;
            }
        };
        uint32_t r = 0;
        if (!outputs) {
            for (; r < cnt; r++) {
                float v[C], out[C], den;
                values(r, v);
                token_update<MODE, RPT, C, false>(sq, sk + r * KS, sw + r * KS, u, v, MODE == kMlstm ? s_gate[buf][0][r] : 0.f,
                                                  MODE == kMlstm ? s_gate[buf][1][r] : 0.f, S, n, out, den);
            }
        }
        for (; r + 8 <= cnt; r += 8) {                       // 8 tokens at a time: one shared reduction, loads run ahead
            float out[C][8], den[8];
#pragma unroll
            for (int i = 0; i < 8; i++) {
                float v[C], o1[C];
                values(r + i, v);
                token_update<MODE, RPT, C, true>(sq + (r + i) * KS, sk + (r + i) * KS, sw + (r + i) * KS, u, v, MODE == kMlstm ? s_gate[buf][0][r + i] : 0.f,
                                                 MODE == kMlstm ? s_gate[buf][1][r + i] : 0.f, S, n, o1, den[i]);
#pragma unroll
                for (int j = 0; j < C; j++) out[j][i] = o1[j];
            }
            const float d = MODE == kMlstm ? reduce8(den, ks) : 0.f;
            float y[C];
#pragma unroll
            for (int j = 0; j < C; j++) {
                y[j] = reduce8(out[j], ks);
                if (MODE == kMlstm) y[j] = mlstm_out(y[j], d, p.qscale, s_gate[buf][2][r + ks]);
                if (MODE == kGla) y[j] *= p.qscale;
            }
            float *at = dst + (size_t)(r + ks) * vpitch;
            if (C == 4 && vec_v) {
                if (col < vdim) *reinterpret_cast<float4 *>(at) = make_float4(y[0], y[1], y[C - 2], y[C - 1]);
            } else {
#pragma unroll
                for (int j = 0; j < C; j++)
                    if (col + j < vdim) at[j] = y[j];
            }
        }
        for (; r < cnt; r++) {
            float v[C], out[C], den;
            values(r, v);
            token_update<MODE, RPT, C, true>(sq + r * KS, sk + r * KS, sw + r * KS, u, v, MODE == kMlstm ? s_gate[buf][0][r] : 0.f,
                                             MODE == kMlstm ? s_gate[buf][1][r] : 0.f, S, n, out, den);
            den = sum8(den);
#pragma unroll
            for (int j = 0; j < C; j++) {
                const float y = sum8(out[j]) * (MODE == kGla ? p.qscale : 1.f);
                if (ks == 0 && col + j < vdim) dst[(size_t)r * vpitch + j] = MODE == kMlstm ? mlstm_out(y, den, p.qscale, s_gate[buf][2][r]) : y;
            }
        }
        if (MODE == kMlstm && t < 32 && c + 1 < chunks) gates(c + 1, buf ^ 1u);
        __syncthreads();
    }
    if (MODE == kMlstm) {
        if (t == 0) { s_end[0] = m; s_end[1] = f_sum; }
        __syncthreads();
    }
    const bool last = row0 + rows == p.rows;
    float *end = last ? p.state : p.segments + seg * stride;
    const bool store = p.phase != 2 || last;             // in phase 2 later segments may still be reading the end states
#pragma unroll
    for (int c = 0; c < C; c++)
        if (store && col + c < vdim) store_keys<RPT>(end + ((size_t)head * vdim + col + c) * kp, ks, kp, S[c]);
    if (store && (MODE == kMlstm || !last)) {
        float *nb = normalizer(p, end, head, block);
        if (t < 8) store_keys<RPT>(nb, ks, kp, n);
        if (MODE == kMlstm && t == 0) {
            nb[kp] = s_end[0];
            if (!last) nb[kp + 1] = s_end[1];
        }
    }
    if (MODE == kWkv && p.shift_state && p.phase != 1 && block == 0 && blockIdx.z == 0) {
        for (uint32_t j = head * kScanThreads + t; j < p.shift_width; j += p.heads * kScanThreads) p.shift_state[j] = p.shift_state[p.shift_width + j];
    }
}

// ---------------------------------------------------------------- one token: decay / gates, recurrence, head norm, gate
constexpr uint32_t kStepThreads = 512, kStepCols = kStepThreads / 8, kStepCluster = 8;

template <int MODE, int RPT, typename OT>
__global__ void __launch_bounds__(kStepThreads) step_kernel(const __grid_constant__ Scan p, const __grid_constant__ HeadGate hg,
                                                            const __grid_constant__ Decay d)
{
    constexpr int KS = RPT * 8;
    extern __shared__ __align__(16) float smem[];        // q, k, w [KS] each; o [vdim]; the decay's low-rank input [rank]
    __shared__ float s_part[kStepThreads / 32], s_gate[3], s_squares;
    const uint32_t t = threadIdx.x, head = blockIdx.x, part = blockIdx.y, parts = gridDim.y, ks = t & 7u, dim = p.dim, vdim = p.vdim, kp = pad4(dim);
    float *sq = smem, *sk = sq + KS, *sw = sk + KS, *so = sw + KS, *s_low = so + vdim;
    float u[RPT], n[RPT];
#pragma unroll
    for (int i = 0; i < RPT; i++) {
        const uint32_t key = (i / 4 * 8 + ks) * 4 + i % 4;
        u[i] = MODE == kWkv && key < dim ? __ldg(p.u + head * dim + key) : 0.f;
        n[i] = 0.f;
    }
    pdl_launch_dependents();
    pdl_wait();
    for (uint32_t i = t; i < (uint32_t)KS; i += kStepThreads) {
        sq[i] = i < dim ? p.q[head * dim + i] : 0.f;
        sk[i] = i < dim ? p.k[head * dim + i] : 0.f;
        sw[i] = 0.f;
    }
    // mlstm: every CTA reads and advances the copies of n and m that belong to its columns
    const uint32_t blocks_per_part = kStepCols / block_cols(dim);
    float *nrow = normalizer(p, p.state, head, part * blocks_per_part);
    if (MODE != kMlstm) {
        const __nv_bfloat16 *w2 = static_cast<const __nv_bfloat16 *>(d.w2);
        const uint32_t rank = d.rank;
        for (uint32_t i = t; i < rank; i += kStepThreads) s_low[i] = decay_input(d.low[i], d.inv_tau);
        __syncthreads();
        for (uint32_t ch = t / 8; ch < ((dim + 3u) & ~3u); ch += kStepCols) {       // a warp covers 4 channels: uniform trip count
            float acc = 0.f;
            if (ch < dim)
                for (uint32_t j = ks; j < rank; j += 8) acc = fmaf(s_low[j], __bfloat162float(w2[(size_t)(head * dim + ch) * rank + j]), acc);
#pragma unroll
            for (int off = 4; off > 0; off >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, off);
            if (ks == 0 && ch < dim) sw[ch] = decay_value(acc + d.w0[head * dim + ch], d.inv_tau);
        }
    } else {
        load_keys<RPT>(nrow, ks, kp, n);
        if (t == 0) {
            const float m0 = nrow[kp], li = p.cap * tanhf(p.gi[head] / p.cap), lf = log_sigmoid(p.cap * tanhf(p.gf[head] / p.cap));
            const float m = fmaxf(lf + m0, li);
            s_gate[0] = expf(lf + m0 - m);
            s_gate[1] = expf(li - m);
            s_gate[2] = m;
        }
    }
    __syncthreads();
    const float a = MODE == kMlstm ? s_gate[0] : 0.f, b = MODE == kMlstm ? s_gate[1] : 0.f, m_new = MODE == kMlstm ? s_gate[2] : 0.f;
    float ss = 0.f, n_out[RPT];
#pragma unroll
    for (int i = 0; i < RPT; i++) n_out[i] = 0.f;
    for (uint32_t c0 = part * kStepCols; c0 < vdim; c0 += parts * kStepCols) {
        const uint32_t col = c0 + t / 8;
        const bool live = col < vdim;
        float *srow = p.state + ((size_t)head * vdim + (live ? col : 0)) * kp;
        float S[1][RPT], nn[RPT], out1[1], den;
        load_keys<RPT>(srow, ks, kp, S[0]);
#pragma unroll
        for (int i = 0; i < RPT; i++) nn[i] = n[i];
        const float v[1] = {live ? p.v[head * vdim + col] : 0.f};
        token_update<MODE, RPT, 1, true>(sq + ks * 4, sk + ks * 4, sw + ks * 4, u, v, a, b, S, nn, out1, den);
        float out = sum8(out1[0]);
        if (MODE == kGla) out *= p.qscale;
        if (MODE == kMlstm) {
            out = mlstm_out(out, sum8(den), p.qscale, expf(-m_new));
#pragma unroll
            for (int i = 0; i < RPT; i++) n_out[i] = nn[i];
        }
        if (live) {
            store_keys<RPT>(srow, ks, kp, S[0]);
            if (ks == 0) { so[col] = out; ss = fmaf(out, out, ss); }
        }
    }
    ss = block_sum(ss, s_part);                          // its barriers also publish so[] and order the reads of n and m
    if (parts > 1) {
        if (t == 0) s_squares = ss;
        cluster_sync();
        ss = 0.f;
        for (uint32_t i = 0; i < parts; i++) ss += cluster_load(&s_squares, i);
        cluster_sync();                                  // no CTA leaves while its sum may still be read
    }
    const float r = 1.0f / sqrtf(ss / (float)vdim + hg.eps);
    OT *dst = static_cast<OT *>(hg.out) + head * vdim;
    for (uint32_t j = t; j < vdim; j += kStepThreads) {
        if (j / kStepCols % parts != part) continue;
        const float g = hg.gate[head * vdim + j], s = sigmoid_f(g);
        dst[j] = from_f32<OT>(so[j] * r * hg.weight[hg.shared ? j : head * vdim + j] * (hg.silu ? g * s : s));
    }
    if (MODE == kMlstm) {
        for (uint32_t blk = t / 8; blk < value_blocks(dim, vdim); blk += kStepCols) {
            if (blk / blocks_per_part % parts != part) continue;
            float *nb = normalizer(p, p.state, head, blk);
            store_keys<RPT>(nb, ks, kp, n_out);
            if (ks == 0) nb[kp] = m_new;
        }
    } else if (p.shift_state && part == 0) {
        for (uint32_t j = head * kStepThreads + t; j < p.shift_width; j += p.heads * kStepThreads) p.shift_state[j] = p.shift_state[p.shift_width + j];
    }
}

// Tokens per segment; rows: no cut.  Segments pay only when two launches of all but one of them are
// shorter than one pass, i.e. from three segments on.
uint32_t segment_length(uint32_t rows, uint32_t heads, uint32_t dim, uint32_t vdim)
{
    const uint32_t ctas = heads * value_blocks(dim, vdim);
    const uint32_t want = std::min(8u, (148u * 3u + ctas - 1) / ctas) + 1;
    if (want < 3 || rows < 256) return rows;
    const uint32_t len = std::max(64u, ((rows + want - 1) / want + 31u) & ~31u);
    return (rows + len - 1) / len < 3 ? rows : len;
}

// Launched without programmatic overlap: few long-running CTAs that would otherwise be packed onto the
// SMs that the preceding kernel happens to leave first.
template <int MODE, int RPT>
int launch_scan_rpt(Scan p, void *workspace, cudaStream_t stream)
{
    constexpr int NA = MODE != kMlstm ? 3 : 2, TC = chunk_tokens<RPT>(), COLS = 16 * thread_cols<RPT>();
    const size_t smem = (size_t)2 * (NA * TC * RPT * 8 + TC * COLS) * sizeof(float);
    if (int rc = allow_smem(scan_kernel<MODE, RPT>, smem)) return rc;
    p.segments = static_cast<float *>(workspace);
    p.seg_len = p.segments ? segment_length(p.rows, p.heads, p.dim, p.vdim) : p.rows;
    p.seg_count = (p.rows + p.seg_len - 1) / p.seg_len;
    dim3 grid(p.heads, value_blocks(p.dim, p.vdim));
    if (p.seg_count == 1) {
        scan_kernel<MODE, RPT><<<grid, kScanThreads, smem, stream>>>(p);
    } else {
        grid.z = p.seg_count - 1;
        p.phase = 1;
        scan_kernel<MODE, RPT><<<grid, kScanThreads, smem, stream>>>(p);
        MGQ_CUDA(cudaGetLastError());
        p.phase = 2;
        scan_kernel<MODE, RPT><<<grid, kScanThreads, smem, stream>>>(p);
    }
    MGQ_CUDA(cudaGetLastError());
    return MGQ_OK;
}

template <int MODE>
int launch_scan(const Scan &p, void *workspace, cudaStream_t stream)
{
    if (p.dim <= 32) return launch_scan_rpt<MODE, 4>(p, workspace, stream);
    if (p.dim <= 64) return launch_scan_rpt<MODE, 8>(p, workspace, stream);
    if (p.dim <= 128) return launch_scan_rpt<MODE, 16>(p, workspace, stream);
    if (p.dim <= kMaxStateDim) return launch_scan_rpt<MODE, 32>(p, workspace, stream);
    return fail(MGQ_ERR_SHAPE, "recurrent heads of %u key dimensions (at most %u)", p.dim, kMaxStateDim);
}

template <int MODE, int RPT>
int launch_step_rpt(const Scan &p, const HeadGate &hg, const Decay &d, cudaStream_t stream)
{
    const size_t smem = (size_t)(3 * RPT * 8 + p.vdim + d.rank) * sizeof(float);
    const uint32_t parts = std::min(kStepCluster, (p.vdim + kStepCols - 1) / kStepCols);
    const dim3 grid(p.heads, parts);
    if (hg.out_bf16) {
        if (int rc = allow_smem(step_kernel<MODE, RPT, __nv_bfloat16>, smem)) return rc;
        return launch_clustered(step_kernel<MODE, RPT, __nv_bfloat16>, grid, dim3(kStepThreads), parts, smem, stream, p, hg, d);
    }
    if (int rc = allow_smem(step_kernel<MODE, RPT, float>, smem)) return rc;
    return launch_clustered(step_kernel<MODE, RPT, float>, grid, dim3(kStepThreads), parts, smem, stream, p, hg, d);
}

template <int MODE>
int launch_step(const Scan &p, const HeadGate &hg, const Decay &d, cudaStream_t stream)
{
    if (p.dim <= 32) return launch_step_rpt<MODE, 4>(p, hg, d, stream);
    if (p.dim <= 64) return launch_step_rpt<MODE, 8>(p, hg, d, stream);
    if (p.dim <= 128) return launch_step_rpt<MODE, 16>(p, hg, d, stream);
    if (p.dim <= kMaxStateDim) return launch_step_rpt<MODE, 32>(p, hg, d, stream);
    return fail(MGQ_ERR_SHAPE, "recurrent heads of %u key dimensions (at most %u)", p.dim, kMaxStateDim);
}

Scan channel_decay_args(const ChannelDecay &a)
{
    Scan p{};
    p.q = a.q; p.k = a.k; p.v = a.v; p.w = a.d.out; p.u = a.u; p.o = a.o; p.state = a.state; p.shift_state = a.shift_state;
    p.rows = a.rows; p.heads = a.heads; p.dim = a.dim; p.vdim = a.vdim; p.shift_width = a.shift_width;
    p.cap = 1.f; p.qscale = a.u ? 1.f : (float)(1.0 / sqrt((double)a.dim));
    return p;
}
Scan mlstm_args(const Mlstm &a)
{
    Scan p{};
    p.q = a.q; p.k = a.k; p.v = a.v; p.gi = a.gi; p.gf = a.gf; p.o = a.o; p.state = a.state;
    p.rows = a.rows; p.heads = a.heads; p.dim = a.dim; p.vdim = a.vdim;
    p.cap = a.cap; p.qscale = (float)(1.0 / sqrt((double)a.dim));
    return p;
}

inline uint32_t blocks_for(size_t n) { return (uint32_t)((n + 255) / 256); }

}  // namespace

int launch_embedding_scaled(const Embedding &a, void *stream)
{
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (a.width % 8 == 0) {
        const dim3 grid(blocks_for((size_t)a.rows * a.width / 8));
        return a.table_bf16 ? launch(embedding_vec_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, a) : launch(embedding_vec_kernel<float>, grid, dim3(256), 0, st, a);
    }
    const dim3 grid(blocks_for((size_t)a.rows * a.width));
    return a.table_bf16 ? launch(embedding_scaled_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, a) : launch(embedding_scaled_kernel<float>, grid, dim3(256), 0, st, a);
}

int launch_norm(const float *x, const float *weight, const uint32_t *index, void *out, bool out_bf16, uint32_t rows, uint32_t src_rows,
                uint32_t cols, float eps, float offset, void *stream)
{
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (out_bf16) return launch(norm_kernel<__nv_bfloat16>, dim3(rows), dim3(256), 0, st, x, weight, index, static_cast<__nv_bfloat16 *>(out), src_rows, cols, eps, offset);
    return launch(norm_kernel<float>, dim3(rows), dim3(256), 0, st, x, weight, index, static_cast<float *>(out), src_rows, cols, eps, offset);
}

int launch_pick_rows(const float *x, const uint32_t *index, float *out, uint32_t rows, uint32_t src_rows, uint32_t cols, void *stream)
{
    return launch(pick_rows_kernel, dim3(blocks_for((size_t)rows * cols)), dim3(256), 0, static_cast<cudaStream_t>(stream), x, index, out, rows, src_rows, cols);
}

int launch_bias_add(const float *x, const float *bias, float *out, uint32_t rows, uint32_t cols, void *stream)
{
    const size_t len = (size_t)rows * cols;
    return launch(bias_add_kernel, dim3(blocks_for(len)), dim3(256), 0, static_cast<cudaStream_t>(stream), x, bias, out, len, cols);
}

int launch_glu(const float *gate, const float *up, void *out, bool out_bf16, size_t len, const Glu &act, void *stream)
{
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (out_bf16) return launch(glu_kernel<__nv_bfloat16>, dim3(blocks_for(len)), dim3(256), 0, st, gate, up, static_cast<__nv_bfloat16 *>(out), len, act);
    return launch(glu_kernel<float>, dim3(blocks_for(len)), dim3(256), 0, st, gate, up, static_cast<float *>(out), len, act);
}

int launch_cast(const float *x, __nv_bfloat16 *out, size_t len, void *stream)
{
    return launch(cast_kernel, dim3(blocks_for(len)), dim3(256), 0, static_cast<cudaStream_t>(stream), x, out, len);
}

int launch_scaled_sum(const float *a, const float *b, float *out, size_t len, float sa, float sb, void *stream)
{
    return launch(scaled_sum_kernel, dim3(blocks_for(len)), dim3(256), 0, static_cast<cudaStream_t>(stream), a, b, out, len, sa, sb);
}

int launch_residual_norm(const ResidualNorm &a, void *stream)
{
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (a.cols % 4) return launch(residual_norm_kernel<1, 4>, dim3(a.rows), dim3(256), 0, st, a);
    if (a.cols <= 1024) return launch(residual_norm_kernel<4, 1>, dim3(a.rows), dim3(256), 0, st, a);
    if (a.cols <= 2048) return launch(residual_norm_kernel<4, 2>, dim3(a.rows), dim3(256), 0, st, a);
    return launch(residual_norm_kernel<4, 4>, dim3(a.rows), dim3(256), 0, st, a);
}

template <typename OT>
static int launch_token_shift_vec(const TokenShift &a, cudaStream_t st)
{
    const uint32_t nv = (a.width + 1023) / 1024, per = a.rows >= 592 ? 4 : 1;
    const dim3 grid((a.rows + per - 1) / per, a.rows == 1 ? nv : 1);
    if (nv <= 1) return launch(token_shift_vec_kernel<OT, 1>, grid, dim3(256), 0, st, a, per);
    if (nv <= 2) return launch(token_shift_vec_kernel<OT, 2>, grid, dim3(256), 0, st, a, per);
    if (nv <= 4) return launch(token_shift_vec_kernel<OT, 4>, grid, dim3(256), 0, st, a, per);
    return launch(token_shift_vec_kernel<OT, 8>, grid, dim3(256), 0, st, a, per);
}

int launch_token_shift(const TokenShift &a, void *stream)
{
    if (a.slots == 0 || a.slots > kMaxShifts) return fail(MGQ_ERR_SHAPE, "token_shift: %u mixes (1..%d)", a.slots, kMaxShifts);
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (a.width % 4 == 0 && a.width <= 8192 && reinterpret_cast<uintptr_t>(a.x) % 16 == 0)
        return a.out_bf16 ? launch_token_shift_vec<__nv_bfloat16>(a, st) : launch_token_shift_vec<float>(a, st);
    if (a.out_bf16) return launch(token_shift_kernel<__nv_bfloat16>, dim3(a.rows), dim3(256), 0, st, a);
    return launch(token_shift_kernel<float>, dim3(a.rows), dim3(256), 0, st, a);
}

int launch_head_gate(const float *o, const HeadGate &hg, uint32_t rows, uint32_t heads, uint32_t dim, void *stream)
{
    const uint32_t total = rows * heads;
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (dim % 4 == 0 && dim <= 512) {
        auto go = [&](auto kernel_f32, auto kernel_bf16, uint32_t lanes) {
            const dim3 grid((uint32_t)(((size_t)total * lanes + 255) / 256));
            return hg.out_bf16 ? launch(kernel_bf16, grid, dim3(256), 0, st, o, hg, total, heads, dim) : launch(kernel_f32, grid, dim3(256), 0, st, o, hg, total, heads, dim);
        };
        if (dim <= 32) return go(head_gate_vec_kernel<float, 8, 1>, head_gate_vec_kernel<__nv_bfloat16, 8, 1>, 8);
        if (dim <= 64) return go(head_gate_vec_kernel<float, 16, 1>, head_gate_vec_kernel<__nv_bfloat16, 16, 1>, 16);
        if (dim <= 128) return go(head_gate_vec_kernel<float, 32, 1>, head_gate_vec_kernel<__nv_bfloat16, 32, 1>, 32);
        return go(head_gate_vec_kernel<float, 32, 4>, head_gate_vec_kernel<__nv_bfloat16, 32, 4>, 32);
    }
    if (hg.out_bf16) return launch(head_gate_kernel<__nv_bfloat16>, dim3((total + 7) / 8), dim3(256), 0, st, o, hg, total, heads, dim);
    return launch(head_gate_kernel<float>, dim3((total + 7) / 8), dim3(256), 0, st, o, hg, total, heads, dim);
}

size_t channel_decay_state_elements(uint32_t heads, uint32_t dim, uint32_t vdim) { return (size_t)heads * vdim * pad4(dim); }
size_t mlstm_state_elements(uint32_t heads, uint32_t dim, uint32_t vdim) { return block_elements(heads, dim, vdim); }
size_t scan_workspace(uint32_t max_rows, uint32_t heads, uint32_t dim, uint32_t vdim)
{
    return max_rows < 256 ? 0 : 8 * block_elements(heads, dim, vdim) * sizeof(float);       // at most 9 segments, the last one ends in the state
}

int launch_decay(const Decay &a, void *stream)
{
    return launch(decay_kernel, dim3((a.channels + kDecayTile - 1) / kDecayTile, (a.rows + kDecayTile - 1) / kDecayTile), dim3(256), 0,
                  static_cast<cudaStream_t>(stream), a);
}

int launch_channel_decay_scan(const ChannelDecay &a, void *stream)
{
    const Scan p = channel_decay_args(a);
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (a.split_products && a.rows >= kPrefillRows) return launch_gla_chunks(a, stream);
    return a.u ? launch_scan<kWkv>(p, a.workspace, st) : launch_scan<kGla>(p, a.workspace, st);
}
int launch_mlstm_scan(const Mlstm &a, void *stream) { return launch_scan<kMlstm>(mlstm_args(a), a.workspace, static_cast<cudaStream_t>(stream)); }
int launch_channel_decay_step(const ChannelDecay &a, const HeadGate &hg, void *stream)
{
    const Scan p = channel_decay_args(a);
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    return a.u ? launch_step<kWkv>(p, hg, a.d, st) : launch_step<kGla>(p, hg, a.d, st);
}
int launch_mlstm_step(const Mlstm &a, const HeadGate &hg, void *stream)
{
    return launch_step<kMlstm>(mlstm_args(a), hg, Decay{}, static_cast<cudaStream_t>(stream));
}

}  // namespace mgq
