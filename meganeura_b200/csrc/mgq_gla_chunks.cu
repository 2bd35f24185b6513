// Gated linear attention over many tokens in chunks of 16 on the tensor cores.
//
// Inside a chunk, with a_t the decays per key channel, L_t = a_1 .. a_t, G_s = a_(s+1) .. a_16 and the
// state S in front of the chunk:
//     o_t = S^T (L_t q_t) + sum_(s <= t) A_ts v_s,      A_ts = sum_d q_t k_s a_(s+1) .. a_t
//     S'  = diag(L_16) S + sum_s (G_s k_s) v_s^T
// Only products of decays appear, never a quotient, so nothing overflows however strong the decay is.
//   gla_prepare_kernel  CTA = chunk x head: the decays from their low-rank projection, then A, L q, G k and L_16
//                       into a record that the next kernel copies as it is
//   gla_chunks_kernel   a warp keeps S^T for 16 value columns and all keys in registers, as f32 accumulators of
//                       mma.sync whose layout is also that of the products' left operand, and walks the chunks;
//                       the records come through a ring of cp.async copies
// State, decays and sums are f32.  Where the state is read it enters as the sum of three bf16, i.e. with all its
// bits; the decayed queries and keys, A and the values as sums of two, three products each: 16 to 17 significant bits
// of numbers whose factors are projections, with the range of f32.  A long portion is cut into segments:
// a first pass leaves the end state of every segment but the last, each started from nothing, gla_combine_kernel
// turns them into the segments' start states, and a second pass runs all segments with outputs.
#include <algorithm>

#include "mgq_mixer.cuh"

namespace mgq {
namespace {

constexpr uint32_t kChunk = 16, kStages = 3, kMaxWarps = 8, kMaxSegs = 16;

// Record of a chunk of a head: G k (high, low parts), L_16, L q (high, low), A (high, low); rows padded for ldmatrix.
template <int D> struct Record {
    static constexpr uint32_t pitch = D + 8, matrix = kChunk * pitch * 2;
    static constexpr uint32_t lam = 2 * matrix, ql = lam + D * 4, a = ql + 2 * matrix, bytes = a + 2 * kChunk * kChunk * 2;
    static constexpr uint32_t state_part = ql;           // what a pass without outputs needs
};

struct Chunks {
    const float *q, *k, *v, *w;                          // w: decays, or null: from d
    Decay d;
    float *o, *state, *segments, *products;              // products: of a segment's decays, [segment][heads][D]
    uint8_t *records;
    uint32_t rows, heads, dim, vdim, chunks;
    uint32_t seg_len, segs, states_only;                 // chunks per segment; the first pass leaves end states only
    float qscale;
};

__device__ __forceinline__ void split2(float x, float y, uint32_t &hi, uint32_t &lo)
{
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const float2 f = __bfloat1622float2(h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
    hi = *reinterpret_cast<const uint32_t *>(&h);
    lo = *reinterpret_cast<const uint32_t *>(&l);
}
__device__ __forceinline__ void split3(float x, float y, uint32_t &hi, uint32_t &mid, uint32_t &lo)
{
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const float2 f = __bfloat1622float2(h);
    hi = *reinterpret_cast<const uint32_t *>(&h);
    split2(x - f.x, y - f.y, mid, lo);
}

template <int D>
__global__ void __launch_bounds__(256) gla_prepare_kernel(const __grid_constant__ Chunks p)
{
    constexpr uint32_t P = D + 4, SLICES = D / 4 < 16 ? D / 4 : 16;
    using R = Record<D>;
    extern __shared__ __align__(16) float smem[];        // q, k, w [16][P], partial sums of A [SLICES][16 t][16 s]
    float *sq = smem, *sk = sq + kChunk * P, *sw = sk + kChunk * P, *sa = sw + kChunk * P;
    const uint32_t t = threadIdx.x, chunk = blockIdx.x, head = blockIdx.y, row0 = chunk * kChunk, kpitch = p.heads * p.dim;
    pdl_launch_dependents();
    pdl_wait();
    // beyond the portion and beyond the head's channels: nothing decays and nothing is added
    if (p.dim % 4 == 0) {
#pragma unroll
        for (uint32_t j = 0; j < (kChunk * D / 4 + 255) / 256; j++) {
            const uint32_t i = t + 256 * j, r = i / (D / 4), d = i % (D / 4) * 4;
            if (i >= kChunk * D / 4) break;
            const bool in = row0 + r < p.rows && d < p.dim;
            const size_t at = (size_t)(row0 + r) * kpitch + head * p.dim + d;
            float4 q = make_float4(0.f, 0.f, 0.f, 0.f), k = q;
            if (in) { q = *reinterpret_cast<const float4 *>(p.q + at); k = *reinterpret_cast<const float4 *>(p.k + at); }
            *reinterpret_cast<float4 *>(sq + r * P + d) = make_float4(q.x * p.qscale, q.y * p.qscale, q.z * p.qscale, q.w * p.qscale);
            *reinterpret_cast<float4 *>(sk + r * P + d) = k;
        }
    } else {
#pragma unroll 4
        for (uint32_t i = t; i < kChunk * D; i += 256) {
            const uint32_t r = i / D, d = i % D;
            const bool in = row0 + r < p.rows && d < p.dim;
            const size_t at = (size_t)(row0 + r) * kpitch + head * p.dim + d;
            sq[r * P + d] = in ? p.q[at] * p.qscale : 0.f;
            sk[r * P + d] = in ? p.k[at] : 0.f;
        }
    }
    if (p.w) {
#pragma unroll 4
        for (uint32_t i = t; i < kChunk * D; i += 256) {
            const uint32_t r = i / D, d = i % D;
            const bool in = row0 + r < p.rows && d < p.dim;
            sw[r * P + d] = in ? p.w[(size_t)(row0 + r) * kpitch + head * p.dim + d] : 1.f;
        }
    } else {
        // thread = channel x a share of the tokens; the low-rank inputs lie where the partial sums of A go later
        constexpr uint32_t GROUPS = 256 / D, PER = kChunk / GROUPS;
        const uint32_t d = t % D, r0 = t / D * PER, ranks = p.d.rank;
        float z[PER];
        for (uint32_t j0 = 0; j0 < ranks; j0 += 128) {
            const uint32_t nj = min(128u, ranks - j0);
            __syncthreads();
            for (uint32_t i = t; i < kChunk * nj; i += 256) {
                const uint32_t r = i / nj, j = i % nj;
                sa[r * 128 + j] = row0 + r < p.rows ? decay_input(p.d.low[(size_t)(row0 + r) * ranks + j0 + j], p.d.inv_tau) : 0.f;
            }
            __syncthreads();
            if (d < p.dim) {
                if (j0 == 0)
#pragma unroll
                    for (int i = 0; i < (int)PER; i++) z[i] = p.d.w0[head * p.dim + d];
                const __nv_bfloat16 *w2 = static_cast<const __nv_bfloat16 *>(p.d.w2) + (size_t)(head * p.dim + d) * ranks + j0;
#pragma unroll 8
                for (uint32_t j = 0; j < nj; j++) {
                    const float x = __bfloat162float(w2[j]);
#pragma unroll
                    for (int i = 0; i < (int)PER; i++) z[i] = fmaf(x, sa[(r0 + i) * 128 + j], z[i]);
                }
            }
        }
#pragma unroll
        for (int i = 0; i < (int)PER; i++) sw[(r0 + i) * P + d] = d < p.dim && row0 + r0 + i < p.rows ? decay_value(z[i], p.d.inv_tau) : 1.f;
    }
    __syncthreads();
    uint8_t *rec = p.records + ((size_t)head * p.chunks + chunk) * R::bytes;
    // A: thread = key token s x a share of the channels; the key decays from token to token
    {
        const uint32_t s = t & 15u, slice = t >> 4;
        float acc[kChunk];
#pragma unroll
        for (int i = 0; i < (int)kChunk; i++) acc[i] = 0.f;
        for (uint32_t d = slice * 4; d < (uint32_t)D; d += 64) {
            const float4 k4 = *reinterpret_cast<const float4 *>(sk + s * P + d);
            float4 r = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int i = 0; i < (int)kChunk; i++) {
                const float4 w4 = *reinterpret_cast<const float4 *>(sw + i * P + d), q4 = *reinterpret_cast<const float4 *>(sq + i * P + d);
                const bool own = (uint32_t)i == s;
                r.x = own ? k4.x : r.x * w4.x; r.y = own ? k4.y : r.y * w4.y; r.z = own ? k4.z : r.z * w4.z; r.w = own ? k4.w : r.w * w4.w;
                acc[i] = fmaf(r.x, q4.x, acc[i]); acc[i] = fmaf(r.y, q4.y, acc[i]); acc[i] = fmaf(r.z, q4.z, acc[i]); acc[i] = fmaf(r.w, q4.w, acc[i]);
            }
        }
        if (slice < SLICES)
#pragma unroll
            for (int i = 0; i < (int)kChunk; i++) sa[(slice * kChunk + i) * kChunk + s] = acc[i];
    }
    // L q by the first half of the threads, G k and L_16 by the second, two channels each
    {
        const uint32_t d = (t & 127u) * 2;
        if (d < (uint32_t)D) {
            float2 f = make_float2(1.f, 1.f);
            if (t < 128) {
#pragma unroll
                for (int i = 0; i < (int)kChunk; i++) {
                    const float2 w2 = *reinterpret_cast<const float2 *>(sw + i * P + d), x = *reinterpret_cast<const float2 *>(sq + i * P + d);
                    f.x *= w2.x; f.y *= w2.y;
                    uint32_t hi, lo;
                    split2(x.x * f.x, x.y * f.y, hi, lo);
                    *reinterpret_cast<uint32_t *>(rec + R::ql + (i * R::pitch + d) * 2) = hi;
                    *reinterpret_cast<uint32_t *>(rec + R::ql + R::matrix + (i * R::pitch + d) * 2) = lo;
                }
            } else {
#pragma unroll
                for (int i = (int)kChunk - 1; i >= 0; i--) {
                    const float2 w2 = *reinterpret_cast<const float2 *>(sw + i * P + d), x = *reinterpret_cast<const float2 *>(sk + i * P + d);
                    uint32_t hi, lo;
                    split2(x.x * f.x, x.y * f.y, hi, lo);
                    *reinterpret_cast<uint32_t *>(rec + (i * R::pitch + d) * 2) = hi;
                    *reinterpret_cast<uint32_t *>(rec + R::matrix + (i * R::pitch + d) * 2) = lo;
                    f.x *= w2.x; f.y *= w2.y;
                }
                *reinterpret_cast<float2 *>(rec + R::lam + d * 4) = f;
            }
        }
    }
    __syncthreads();
    if (t < 128) {                                       // two neighbouring keys of one query
        float2 x = make_float2(0.f, 0.f);
#pragma unroll
        for (int i = 0; i < (int)SLICES; i++) {
            const float2 y = *reinterpret_cast<const float2 *>(sa + i * kChunk * kChunk + 2 * t);
            x.x += y.x; x.y += y.y;
        }
        uint32_t hi, lo;
        split2(x.x, x.y, hi, lo);
        *reinterpret_cast<uint32_t *>(rec + R::a + 4 * t) = hi;
        *reinterpret_cast<uint32_t *>(rec + R::a + kChunk * kChunk * 2 + 4 * t) = lo;
    }
}

__device__ __forceinline__ uint32_t smem_addr(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }
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
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// CTA = head (x) x value columns (y), 16 per warp, x segment (z).
template <int D>
__global__ void __launch_bounds__(256, 1) gla_chunks_kernel(const __grid_constant__ Chunks p)
{
    using R = Record<D>;
    extern __shared__ __align__(16) uint8_t ring[];      // kStages records
    __shared__ float s_f[D];                             // product of the decays so far (first pass)
    const uint32_t t = threadIdx.x, threads = blockDim.x, lane = t & 31u, warp = t >> 5, g = lane >> 2, tq = lane & 3u;
    const uint32_t head = blockIdx.x, v0 = (blockIdx.y * (threads >> 5) + warp) * 16, kp = (p.dim + 3u) & ~3u, vpitch = p.heads * p.vdim;
    const uint32_t seg = blockIdx.z, c0 = seg * p.seg_len, c1 = min(c0 + p.seg_len, p.chunks);
    const bool outputs = !p.states_only;
    const uint32_t vr[2] = {v0 + g, v0 + g + 8};         // this thread's value columns
    const bool live[2] = {vr[0] < p.vdim, vr[1] < p.vdim};
    pdl_launch_dependents();
    pdl_wait();
    const uint8_t *records = p.records + (size_t)head * p.chunks * R::bytes;
    auto stage = [&](uint32_t c) {                       // always one commit
        if (c < c1) {
            const uint8_t *src = records + (size_t)c * R::bytes;
            const uint32_t dst = smem_addr(ring + (c - c0) % kStages * R::bytes), bytes = outputs ? R::bytes : R::state_part;
            for (uint32_t i = t * 16; i < bytes; i += threads * 16)
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(dst + i), "l"(src + i) : "memory");
        }
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };
    stage(c0);
    stage(c0 + 1);
    const float *vbase = p.v + head * p.vdim;
    float v[8];
    auto load_values = [&](uint32_t c) {                 // [token pair low / high half][column], two tokens each
#pragma unroll
        for (int h = 0; h < 2; h++)
#pragma unroll
            for (int i = 0; i < 2; i++)
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    const uint32_t row = c * kChunk + h * 8 + tq * 2 + e;
                    v[(h * 2 + i) * 2 + e] = c < c1 && row < p.rows && live[i] ? vbase[(size_t)row * vpitch + vr[i]] : 0.f;
                }
    };
    load_values(c0);

    // S^T: rows are value columns, columns are keys
    float S[D / 8][4];
#pragma unroll
    for (int n = 0; n < D / 8; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) S[n][e] = 0.f;
    if (seg == 0 || outputs) {                           // start state: the sequence's, or what the combination left
        const bool own = seg == 0 && (p.segs == 1 || !outputs);
        const uint32_t slot = seg == 0 ? p.segs - 1 : seg - 1, pitch = own ? kp : D;
        const float *start = own ? p.state + (size_t)head * p.vdim * kp : p.segments + ((size_t)slot * p.heads + head) * p.vdim * D;
#pragma unroll
        for (int n = 0; n < D / 8; n++)
#pragma unroll
            for (int i = 0; i < 2; i++) {
                const uint32_t d = n * 8 + tq * 2;
                if (d < pitch && live[i]) {
                    const float2 x = *reinterpret_cast<const float2 *>(start + (size_t)vr[i] * pitch + d);
                    S[n][2 * i] = x.x; S[n][2 * i + 1] = x.y;
                }
            }
    }

    const bool product = !outputs && blockIdx.y == 0;
    if (product)
        for (uint32_t d = t; d < (uint32_t)D; d += threads) s_f[d] = 1.f;      // a thread only ever touches its own entries
    const uint32_t q_off = R::ql + (((lane & 7u) + (lane >> 4) * 8) * R::pitch + ((lane >> 3) & 1u) * 8) * 2;
    const uint32_t k_off = (((lane & 7u) + ((lane >> 3) & 1u) * 8) * R::pitch + (lane >> 4) * 8) * 2;
    for (uint32_t c = c0; c < c1; c++) {
        asm volatile("cp.async.wait_group 1;\n" ::: "memory");
        __syncthreads();                                 // everyone's copies, and everyone has left the buffer that is filled now
        stage(c + 2);
        const uint8_t *rec = ring + (c - c0) % kStages * R::bytes;
        const uint32_t base = smem_addr(rec);
        uint32_t vh[4], vl[4];                           // V^T as left operand: rows value columns, columns tokens
#pragma unroll
        for (int i = 0; i < 4; i++) split2(v[2 * i], v[2 * i + 1], vh[i], vl[i]);
        load_values(c + 1);
        float o[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};          // o^T: rows value columns, columns tokens
#pragma unroll
        for (int j = 0; j < D / 16; j++) {
            uint32_t sh[4], sm[4], sl[4], qh[4], ql[4], kh[4], kl[4];
            if (outputs) {
                split3(S[2 * j][0], S[2 * j][1], sh[0], sm[0], sl[0]);
                split3(S[2 * j][2], S[2 * j][3], sh[1], sm[1], sl[1]);
                split3(S[2 * j + 1][0], S[2 * j + 1][1], sh[2], sm[2], sl[2]);
                split3(S[2 * j + 1][2], S[2 * j + 1][3], sh[3], sm[3], sl[3]);
                ldmatrix4(base + q_off + j * 32, qh);
                ldmatrix4(base + q_off + R::matrix + j * 32, ql);
            }
            ldmatrix4_t(base + k_off + j * 32, kh);
            ldmatrix4_t(base + k_off + R::matrix + j * 32, kl);
#pragma unroll
            for (int n = 0; n < 2; n++) {
                const float2 f = *reinterpret_cast<const float2 *>(rec + R::lam + (j * 16 + n * 8 + tq * 2) * 4);
                float (&x)[4] = S[2 * j + n];
                x[0] *= f.x; x[1] *= f.y; x[2] *= f.x; x[3] *= f.y;
            }
            // small products first; the sums are independent of each other
#pragma unroll
            for (int part = 0; part < 5; part++) {
                const uint32_t (&sa)[4] = part == 0 ? sl : part == 1 || part == 3 ? sm : sh, (&qb)[4] = part == 1 || part == 2 ? ql : qh;
                if (outputs) {
                    mma16816(o[0], sa, qb[0], qb[1]);
                    mma16816(o[1], sa, qb[2], qb[3]);
                }
                if (part >= 3) continue;
                const uint32_t (&va)[4] = part == 1 ? vl : vh, (&kb)[4] = part == 0 ? kl : kh;
                mma16816(S[2 * j], va, kb[0], kb[1]);
                mma16816(S[2 * j + 1], va, kb[2], kb[3]);
            }
        }
        if (product)
            for (uint32_t d = t; d < (uint32_t)D; d += threads) s_f[d] *= *reinterpret_cast<const float *>(rec + R::lam + d * 4);
        if (!outputs) continue;
#pragma unroll
        for (int n = 0; n < 2; n++) {                    // tokens n * 8 + g as columns, keys of the chunk as the sum
            const uint8_t *a = rec + R::a + ((n * 8 + g) * kChunk + tq * 2) * 2;
            const uint32_t ah0 = *reinterpret_cast<const uint32_t *>(a), ah1 = *reinterpret_cast<const uint32_t *>(a + 16);
            const uint32_t al0 = *reinterpret_cast<const uint32_t *>(a + kChunk * kChunk * 2), al1 = *reinterpret_cast<const uint32_t *>(a + kChunk * kChunk * 2 + 16);
            mma16816(o[n], vh, al0, al1);
            mma16816(o[n], vl, ah0, ah1);
            mma16816(o[n], vh, ah0, ah1);
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const uint32_t row = c * kChunk + n * 8 + tq * 2 + (e & 1);
                if (row < p.rows && live[e >> 1]) p.o[(size_t)row * vpitch + head * p.vdim + vr[e >> 1]] = o[n][e];
            }
        }
    }
    if (outputs && c1 != p.chunks) return;
    if (product)
        for (uint32_t d = t; d < (uint32_t)D; d += threads) p.products[((size_t)seg * p.heads + head) * D + d] = s_f[d];
#pragma unroll
    for (int n = 0; n < D / 8; n++)
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const uint32_t d = n * 8 + tq * 2;
            if (!live[i]) continue;
            const float2 x = make_float2(S[n][2 * i], S[n][2 * i + 1]);
            if (!outputs)    *reinterpret_cast<float2 *>(p.segments + (((size_t)seg * p.heads + head) * p.vdim + vr[i]) * D + d) = x;
            else if (d < kp) *reinterpret_cast<float2 *>(p.state + ((size_t)head * p.vdim + vr[i]) * kp + d) = x;
        }
}

// End states of segments that started from nothing (the first one: from the state) -> states behind them, in place.
// The last slot receives a copy of the sequence's state, which the last segment of the second pass overwrites.
// CTA = head x kCombineCols value columns; thread = 4 keys of a share of the columns.
constexpr uint32_t kCombineCols = 16;
template <int D>
__global__ void __launch_bounds__(256) gla_combine_kernel(const __grid_constant__ Chunks p)
{
    const uint32_t t = threadIdx.x, head = blockIdx.x, v0 = blockIdx.y * kCombineCols;
    pdl_launch_dependents();
    pdl_wait();
    const size_t step = (size_t)p.heads * p.vdim * D;
    const uint32_t kp = (p.dim + 3u) & ~3u;
    for (uint32_t i = t; i < kCombineCols * D / 4; i += 256) {
        const uint32_t v = v0 + i / (D / 4), d = i % (D / 4) * 4;
        if (v >= p.vdim) break;
        float *at = p.segments + ((size_t)head * p.vdim + v) * D + d;
        float4 S = *reinterpret_cast<const float4 *>(at);
        *reinterpret_cast<float4 *>(at + (p.segs - 1) * step) =
            d < kp ? *reinterpret_cast<const float4 *>(p.state + ((size_t)head * p.vdim + v) * kp + d) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
        for (uint32_t s = 1; s + 1 < p.segs; s++) {
            const float4 x = *reinterpret_cast<const float4 *>(at + s * step), f = *reinterpret_cast<const float4 *>(p.products + ((size_t)s * p.heads + head) * D + d);
            S = make_float4(fmaf(f.x, S.x, x.x), fmaf(f.y, S.y, x.y), fmaf(f.z, S.z, x.z), fmaf(f.w, S.w, x.w));
            *reinterpret_cast<float4 *>(at + s * step) = S;
        }
    }
}

uint32_t padded(uint32_t dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 128 ? 128 : 256; }
uint32_t warps_for(uint32_t vdim) { return std::min(kMaxWarps, (vdim + 15) / 16); }
size_t align256(size_t n) { return (n + 255) & ~(size_t)255; }
size_t record_bytes(uint32_t dim)
{
    const uint32_t d = padded(dim);
    return d == 32 ? Record<32>::bytes : d == 64 ? Record<64>::bytes : d == 128 ? Record<128>::bytes : Record<256>::bytes;
}

// Chunks per segment; all of them: one pass.  Two passes pay from three segments on.
uint32_t segment_chunks(uint32_t chunks, uint32_t heads, uint32_t vdim)
{
    const uint32_t w = warps_for(vdim), ctas = heads * ((vdim + 16 * w - 1) / (16 * w)), want = std::min(kMaxSegs, 148u / ctas);
    if (want < 3 || chunks < 12) return chunks;
    const uint32_t len = std::max(4u, (chunks + want - 1) / want);
    return (chunks + len - 1) / len < 3 ? chunks : len;
}

template <int D>
int launch_sized(Chunks p, cudaStream_t st)
{
    const size_t prep = (size_t)(3 * kChunk * (D + 4) + std::max(std::min(D / 4, 16) * kChunk * kChunk, kChunk * 128)) * 4, smem = (size_t)kStages * Record<D>::bytes;
    if (int rc = allow_smem(gla_prepare_kernel<D>, prep)) return rc;
    if (int rc = allow_smem(gla_chunks_kernel<D>, smem)) return rc;
    if (int rc = launch(gla_prepare_kernel<D>, dim3(p.chunks, p.heads), dim3(256), prep, st, p)) return rc;
    const uint32_t w = warps_for(p.vdim);
    dim3 grid(p.heads, (p.vdim + 16 * w - 1) / (16 * w), p.segs);
    if (p.segs > 1) {
        grid.z = p.segs - 1;
        p.states_only = 1;
        if (int rc = launch(gla_chunks_kernel<D>, grid, dim3(w * 32), smem, st, p)) return rc;
        if (int rc = launch(gla_combine_kernel<D>, dim3(p.heads, (p.vdim + kCombineCols - 1) / kCombineCols), dim3(256), 0, st, p)) return rc;
        grid.z = p.segs;
        p.states_only = 0;
    }
    return launch(gla_chunks_kernel<D>, grid, dim3(w * 32), smem, st, p);
}

}  // namespace

size_t gla_chunks_workspace(uint32_t max_rows, uint32_t heads, uint32_t dim, uint32_t vdim)
{
    if (max_rows < kPrefillRows) return 0;
    const size_t chunks = (max_rows + kChunk - 1) / kChunk;
    return align256(chunks * heads * record_bytes(dim)) + (size_t)kMaxSegs * heads * (vdim + 1) * padded(dim) * 4;
}

int launch_gla_chunks(const ChannelDecay &a, void *stream)
{
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (a.u || a.dim > kMaxStateDim || !a.workspace) return fail(MGQ_ERR_STATE, "gla chunks: not this recurrence");
    Chunks p{};
    p.q = a.q; p.k = a.k; p.v = a.v; p.w = a.decay_pending ? nullptr : a.d.out; p.d = a.d; p.o = a.o; p.state = a.state;
    p.rows = a.rows; p.heads = a.heads; p.dim = a.dim; p.vdim = a.vdim; p.chunks = (a.rows + kChunk - 1) / kChunk;
    p.records = static_cast<uint8_t *>(a.workspace);
    p.segments = reinterpret_cast<float *>(p.records + align256((size_t)p.chunks * a.heads * record_bytes(a.dim)));
    p.products = p.segments + (size_t)kMaxSegs * a.heads * a.vdim * padded(a.dim);
    p.seg_len = segment_chunks(p.chunks, a.heads, a.vdim);
    p.segs = (p.chunks + p.seg_len - 1) / p.seg_len;
    p.qscale = (float)(1.0 / sqrt((double)a.dim));
    switch (padded(a.dim)) {
        case 32: return launch_sized<32>(p, st);
        case 64: return launch_sized<64>(p, st);
        case 128: return launch_sized<128>(p, st);
        default: return launch_sized<256>(p, st);
    }
}

}  // namespace mgq
