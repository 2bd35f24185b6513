// Softmax attention for many rows (a prompt's portion) over f16 keys and values: a blockwise exact softmax,
// CTA = one head x 128 query rows (8 warps x 16 rows) x up to 128 value columns, 64 keys per tile, three
// cp.async stages, tensor-core products with f32 accumulation.  Query heads may share key / value heads.
//
// Latent attention, bf16 cache: the keys W_uk c and values W_uv c of all live cache rows are expanded once
// per step by the tcgen05 linear kernel (ring order, f16).  The rotated key part, shared by the heads, is kept once.
// Scores, maxima, sums and weights are f32.  The operands of the products are f16, not bf16: all are of
// moderate size (a clamp guards the range), and with 11 significant bits the result stays close to the
// absorbed form, which keeps the query in f32, so it hardly matters how a prompt is cut.  Only tiles that some row of the
// CTA can see are visited; positions map to ring rows by position % slots.
#include "mgq_linear.cuh"
#include "mgq_mixer.cuh"

namespace mgq {
namespace {

constexpr uint32_t BM = 128, BN = 64, kStages = 3, kThreads = 256;

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
__device__ __forceinline__ __half to_half(float x) { return from_f32<__half>(x); }

// The shared rotated key parts of the live cache rows as f16.
__global__ void rotated_half_kernel(const __nv_bfloat16 *cache, const uint32_t *pos, __half *out, uint32_t rows, uint32_t slots, uint32_t rank, uint32_t rot)
{
    const uint32_t i = blockIdx.x * 256u + threadIdx.x;
    pdl_launch_dependents();
    pdl_wait();
    if (i >= min(slots, pos[0] + rows) * rot) return;
    const uint32_t slot = i / rot;
    out[i] = to_half(__bfloat162float(cache[(size_t)slot * (rank + rot) + rank + i - slot * rot]));
}

struct Prefill {
    const float *q, *freq;
    const __half *keys, *values, *rotated;          // [slots, kv_heads * dim], [slots, kv_heads * vdim], [slots, rot]
    const uint32_t *pos;
    const float *gate;
    void *out;
    uint32_t rows, heads, kv_heads, dim, rot, vdim, slots, window;
    float scale_log2;                               // scale * log2(e)
    uint32_t out_bf16, silu;
};

// DK: dim + rot, DV: value columns of the CTA (blockIdx.z: which), both rounded up to a multiple of 16.
template <int DK, int DV>
__global__ void __launch_bounds__(kThreads, 1) prefill_attention_kernel(const __grid_constant__ Prefill p)
{
    constexpr int PK = DK + 8, PV = DV + 8;          // row pitch in elements: an odd number of 16-byte pieces
    extern __shared__ __align__(16) __half sm[];
    __half *s_q = sm, *s_k = s_q + BM * PK, *s_v = s_k + kStages * BN * PK;
    const uint32_t t = threadIdx.x, lane = t & 31u, warp = t >> 5, head = blockIdx.x;
    const uint32_t kv_head = head / (p.heads / p.kv_heads), v0 = blockIdx.z * DV, vcols = min(p.vdim - v0, (uint32_t)DV);
    const uint32_t row0 = (gridDim.y - 1 - blockIdx.y) * BM, dk = p.dim + p.rot;      // longest rows first
    pdl_launch_dependents();
    // zero padding columns (they meet in products), and query rows that do not exist
    const __half zero = __float2half_rn(0.f);
    if (dk < DK)
        for (uint32_t i = t; i < (BM + kStages * BN) * (DK - dk); i += kThreads) s_q[i / (DK - dk) * PK + dk + i % (DK - dk)] = zero;
    if (vcols < DV)
        for (uint32_t i = t; i < kStages * BN * (DV - vcols); i += kThreads) s_v[i / (DV - vcols) * PV + vcols + i % (DV - vcols)] = zero;
    for (uint32_t r = p.rows - row0; r < BM; r++)
        for (uint32_t j = t; j < dk; j += kThreads) s_q[r * PK + j] = zero;
    pdl_wait();
    const uint32_t pos0 = p.pos[0], first = pos0 + row0, last = pos0 + min(row0 + BM, p.rows) - 1;
    const uint32_t lo = first + 1 > p.window ? first + 1 - p.window : 0u, tiles = (last - lo) / BN + 1;
    __syncthreads();

    auto stage = [&](uint32_t tile, uint32_t buf) {
        const uint32_t kt = lo + tile * BN;
        const uint32_t kb = smem_addr(s_k + buf * BN * PK), vb = smem_addr(s_v + buf * BN * PV);
        const uint32_t per_k = p.dim / 8, per_r = p.rot / 8, per_v = vcols / 8;
        const uint32_t r = t >> 2, part = t & 3u;                         // four threads per key row
        const size_t slot = min(kt + r, last) % p.slots;                  // beyond the last key: a valid row, masked below
        const __half *ksrc = p.keys + (slot * p.kv_heads + kv_head) * p.dim, *rsrc = p.rotated + slot * p.rot,
                            *vsrc = p.values + (slot * p.kv_heads + kv_head) * p.vdim + v0;
        for (uint32_t c = part; c < per_k; c += 4) cp_async16(kb + (r * PK + c * 8) * 2, ksrc + c * 8);
        for (uint32_t c = part; c < per_r; c += 4) cp_async16(kb + (r * PK + p.dim + c * 8) * 2, rsrc + c * 8);
        for (uint32_t c = part; c < per_v; c += 4) cp_async16(vb + (r * PV + c * 8) * 2, vsrc + c * 8);
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };
    stage(0, 0);
    if (tiles > 1) stage(1, 1);
    else asm volatile("cp.async.commit_group;\n" ::: "memory");

    // queries: unrotated part as it is, rotated part turned by its position
    {
        const uint32_t half = p.rot / 2;
        const size_t pitch = (size_t)p.heads * dk;
        const uint32_t n = min(BM, p.rows - row0), d4 = p.dim / 4;
        const float *base = p.q + (size_t)row0 * pitch + head * dk;
#pragma unroll 8
        for (uint32_t i = t; i < n * d4; i += kThreads) {
            const uint32_t r = i / d4, j = (i - r * d4) * 4;
            const float4 v = *reinterpret_cast<const float4 *>(base + r * pitch + j);
            __half2 *dst = reinterpret_cast<__half2 *>(s_q + r * PK + j);
            dst[0] = __halves2half2(to_half(v.x), to_half(v.y));
            dst[1] = __halves2half2(to_half(v.z), to_half(v.w));
        }
#pragma unroll 4
        for (uint32_t i = t; i < n * half; i += kThreads) {
            const uint32_t r = i / half, j = i - r * half;
            const float *src = base + r * pitch + p.dim;
            const float u = src[j], v = src[half + j];
            float sn, cs;
            sincosf((float)(first + r) * p.freq[j], &sn, &cs);
            s_q[r * PK + p.dim + j] = to_half(u * cs - v * sn);
            s_q[r * PK + p.dim + half + j] = to_half(v * cs + u * sn);
        }
    }
    float o[DV / 8][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
    for (int n = 0; n < DV / 8; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) o[n][e] = 0.f;
    const uint32_t qrow = warp * 16 + lane / 4;                          // this thread's rows: qrow, qrow + 8
    const uint32_t qp[2] = {first + qrow, first + qrow + 8};
    const uint32_t a_addr = smem_addr(s_q + (warp * 16 + (lane & 7u) + ((lane >> 3) & 1u) * 8) * PK + (lane >> 4) * 8);
    const uint32_t b_off = (((lane & 7u) + (lane >> 4) * 8) * PK + ((lane >> 3) & 1u) * 8) * 2;
    const uint32_t v_off = (((lane & 7u) + ((lane >> 3) & 1u) * 8) * PV + (lane >> 4) * 8) * 2;

    for (uint32_t tile = 0; tile < tiles; tile++) {
        const uint32_t buf = tile % kStages, kt = lo + tile * BN;
        asm volatile("cp.async.wait_group 1;\n" ::: "memory");           // one group per tile, the next one may be in flight
        __syncthreads();                                                 // and every warp has left the buffer that is filled now
        if (tile + 2 < tiles) stage(tile + 2, (tile + 2) % kStages);
        else asm volatile("cp.async.commit_group;\n" ::: "memory");
        const uint32_t w_first = first + warp * 16, w_last = w_first + 15;
        if (kt > w_last || kt + BN - 1 + p.window <= w_first) continue;  // no row of this warp sees the tile
        const uint32_t kb = smem_addr(s_k + buf * BN * PK) + b_off, vb = smem_addr(s_v + buf * BN * PV) + v_off;
        float s[BN / 8][4];
#pragma unroll
        for (int n = 0; n < (int)BN / 8; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) s[n][e] = 0.f;
#pragma unroll
        for (int kk = 0; kk < DK / 16; kk++) {
            uint32_t a[4];
            ldmatrix4(a_addr + kk * 32, a);
#pragma unroll
            for (int n = 0; n < (int)BN / 16; n++) {
                uint32_t b[4];
                ldmatrix4(kb + (n * 16 * PK + kk * 16) * 2, b);
                mma16816(s[2 * n], a, b[0], b[1]);
                mma16816(s[2 * n + 1], a, b[2], b[3]);
            }
        }
        // mask only where the tile crosses the diagonal or a row's window edge
        const bool edge = kt + BN - 1 > w_first || kt + p.window <= w_last;
#pragma unroll
        for (int h = 0; h < 2; h++) {
            float mx = -INFINITY;
#pragma unroll
            for (int n = 0; n < (int)BN / 8; n++)
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    float &x = s[n][2 * h + e];
                    x *= p.scale_log2;
                    const uint32_t key = kt + n * 8 + (lane & 3u) * 2 + e;
                    if (edge && !(key <= qp[h] && key + p.window > qp[h])) x = -INFINITY;
                    mx = fmaxf(mx, x);
                }
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
            const float m_new = fmaxf(m[h], mx), base = m_new == -INFINITY ? 0.f : m_new;
            const float corr = exp2f(m[h] - base);        // nothing seen yet: exp2(-inf) = 0
            m[h] = m_new;
            float sum = 0.f;
#pragma unroll
            for (int n = 0; n < (int)BN / 8; n++)
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    float &x = s[n][2 * h + e];
                    x = exp2f(x - base);
                    sum += x;
                }
            l[h] = l[h] * corr + sum;
#pragma unroll
            for (int n = 0; n < DV / 8; n++) { o[n][2 * h] *= corr; o[n][2 * h + 1] *= corr; }
        }
#pragma unroll
        for (int kk = 0; kk < (int)BN / 16; kk++) {
            uint32_t w[4];
#pragma unroll
            for (int j = 0; j < 4; j++) w[j] = pack2(s[2 * kk + j / 2][(j & 1) * 2], s[2 * kk + j / 2][(j & 1) * 2 + 1]);
#pragma unroll
            for (int n = 0; n < DV / 16; n++) {
                uint32_t b[4];
                ldmatrix4_t(vb + (kk * 16 * PV + n * 16) * 2, b);
                mma16816(o[2 * n], w, b[0], b[1]);
                mma16816(o[2 * n + 1], w, b[2], b[3]);
            }
        }
    }
#pragma unroll
    for (int h = 0; h < 2; h++) {
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 1);
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 2);
        const uint32_t row = row0 + qrow + h * 8;
        if (row >= p.rows) continue;
        const float inv = 1.0f / l[h];
        const size_t base = ((size_t)row * p.heads + head) * p.vdim + v0;
#pragma unroll
        for (int n = 0; n < DV / 8; n++) {
            const uint32_t v = n * 8 + (lane & 3u) * 2;
            if (v >= vcols) break;
            float x = o[n][2 * h] * inv, y = o[n][2 * h + 1] * inv;
            if (p.gate) {
                const float2 g = *reinterpret_cast<const float2 *>(p.gate + base + v);
                x *= sigmoid_f(g.x) * (p.silu ? g.x : 1.f);
                y *= sigmoid_f(g.y) * (p.silu ? g.y : 1.f);
            }
            if (p.out_bf16) *reinterpret_cast<__nv_bfloat162 *>(static_cast<__nv_bfloat16 *>(p.out) + base + v) = __floats2bfloat162_rn(x, y);
            else            *reinterpret_cast<float2 *>(static_cast<float *>(p.out) + base + v) = make_float2(x, y);
        }
    }
}

template <int DK, int DV>
int launch_prefill(const Prefill &p, cudaStream_t st)
{
    const size_t smem = ((size_t)(BM + kStages * BN) * (DK + 8) + (size_t)kStages * BN * (DV + 8)) * 2;
    if (int rc = allow_smem(prefill_attention_kernel<DK, DV>, smem)) return rc;
    return launch(prefill_attention_kernel<DK, DV>, dim3(p.heads, (p.rows + BM - 1) / BM, (p.vdim + DV - 1) / DV), dim3(kThreads), smem, st, p);
}

template <int DK>
int launch_prefill_v(const Prefill &p, cudaStream_t st)
{
    if (p.vdim <= 64) return launch_prefill<DK, 64>(p, st);
    return launch_prefill<DK, 128>(p, st);
}

int launch_prefill_sized(const Prefill &p, cudaStream_t st)
{
    const uint32_t dk = p.dim + p.rot;
    if (dk <= 64) return launch_prefill_v<64>(p, st);
    if (dk <= 96) return launch_prefill_v<96>(p, st);
    if (dk <= 128) return launch_prefill_v<128>(p, st);
    if (dk <= 192) return launch_prefill_v<192>(p, st);
    return launch_prefill_v<256>(p, st);
}

void set_output(Prefill &p, const HeadGate *gate, float *o)
{
    p.gate = gate ? gate->gate : nullptr;
    p.out = gate ? gate->out : o;
    p.out_bf16 = gate && gate->out_bf16;
    p.silu = gate && gate->silu;
}

size_t align256(size_t n) { return (n + 255) & ~(size_t)255; }

}  // namespace

bool latent_prefill_eligible(uint32_t dim, uint32_t rot_dim, uint32_t vdim, uint32_t rank, bool cache_bf16)
{
    return cache_bf16 && dim % 8 == 0 && rot_dim % 8 == 0 && vdim % 8 == 0 && rank % 8 == 0 && dim + rot_dim <= 256;
}

size_t latent_prefill_workspace(uint32_t heads, uint32_t dim, uint32_t rot_dim, uint32_t vdim, uint32_t slots)
{
    return align256((size_t)slots * heads * dim * 2) + align256((size_t)slots * heads * vdim * 2) + align256((size_t)slots * rot_dim * 2);
}

int launch_latent_prefill(const LatentAttention &a, void *stream)
{
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    uint8_t *ws = static_cast<uint8_t *>(a.workspace);
    __half *keys = reinterpret_cast<__half *>(ws);
    ws += align256((size_t)a.slots * a.heads * a.dim * 2);
    __half *values = reinterpret_cast<__half *>(ws);
    ws += align256((size_t)a.slots * a.heads * a.vdim * 2);
    __half *rotated = reinterpret_cast<__half *>(ws);
    const __nv_bfloat16 *cache = static_cast<const __nv_bfloat16 *>(a.cache);
    if (a.rot_dim)
        if (int rc = launch(rotated_half_kernel, dim3((uint32_t)(((size_t)a.slots * a.rot_dim + 255) / 256)), dim3(256), 0, st, cache, a.pos, rotated, a.rows, a.slots, a.rank, a.rot_dim)) return rc;
    LinearGroup g{};
    g.count = 2; g.m = a.slots; g.lda = a.rank + a.rot_dim;
    g.a_bf16 = 1; g.out_f16 = 1; g.live = a.pos; g.live_add = a.rows;
    g.seg[0].a = g.seg[1].a = a.cache;
    g.seg[0].k = g.seg[1].k = a.rank;
    g.seg[0].w = a.uk; g.seg[0].out = keys; g.seg[0].n = a.heads * a.dim;
    g.seg[1].w = a.uv; g.seg[1].out = values; g.seg[1].n = a.heads * a.vdim;
    if (int rc = launch_linear_tc(g, stream)) return rc;
    Prefill p{};
    p.q = a.q; p.freq = a.freq; p.keys = keys; p.values = values; p.rotated = rotated; p.pos = a.pos;
    set_output(p, a.gate, a.o);
    p.rows = a.rows; p.heads = p.kv_heads = a.heads; p.dim = a.dim; p.rot = a.rot_dim; p.vdim = a.vdim; p.slots = a.slots; p.window = a.window;
    p.scale_log2 = a.scale * 1.4426950408889634f;
    return launch_prefill_sized(p, st);
}

bool attention_prefill_eligible(const Attention &a) { return a.half && a.rows >= kPrefillRows && a.dim % 8 == 0 && a.vdim % 8 == 0 && a.dim <= 256; }

int launch_attention_prefill(const Attention &a, void *stream)
{
    Prefill p{};
    p.q = a.q; p.keys = static_cast<const __half *>(a.keys); p.values = static_cast<const __half *>(a.values); p.pos = a.pos;
    set_output(p, a.gate, a.o);
    p.rows = a.rows; p.heads = a.heads; p.kv_heads = a.kv_heads; p.dim = a.dim; p.vdim = a.vdim; p.slots = a.slots;
    p.window = 1u << 30;                                 // no position is that far away
    p.scale_log2 = a.scale * 1.4426950408889634f;
    return launch_prefill_sized(p, static_cast<cudaStream_t>(stream));
}

}  // namespace mgq
