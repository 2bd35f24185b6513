// Operators of decoders with recurrent, softmax- and latent-attention mixers (mgq_mixer_ops.cu,
// mgq_attention.cu, mgq_latent_attention.cu, mgq_prefill_attention.cu).  All pointers are device pointers; activations are f32 unless an
// argument says bf16; `rows` consecutive tokens of one sequence.
#pragma once
#include "mgq_launch.cuh"

namespace mgq {

constexpr int kMaxShifts = 8;
constexpr uint32_t kMaxStateDim = 256;         // key dimensions of a recurrent head
constexpr uint32_t kPrefillRows = 64;          // from here on a step takes the kernels for many rows

// out[r] = table[ids[r]] * scale (+ sinusoidal vector of position pos + r); copy: a second, bf16 output or null.
// sinusoid: (width + 1) / 2 frequencies as sums of two f32 (null: no position vector); column 2i is the sine
// and column 2i + 1 the cosine of position * frequency i.
struct Embedding {
    const uint32_t *ids, *pos;
    const void *table;
    const float2 *sinusoid;
    float *out;
    __nv_bfloat16 *copy;
    uint32_t rows, width, vocab;
    float scale;
    bool table_bf16;
};
int launch_embedding_scaled(const Embedding &a, void *stream);
// out[r] = unit_rms(x[index ? index[r] : r]) * (offset + weight)
int launch_norm(const float *x, const float *weight, const uint32_t *index, void *out, bool out_bf16, uint32_t rows, uint32_t src_rows,
                uint32_t cols, float eps, float offset, void *stream);
int launch_pick_rows(const float *x, const uint32_t *index, float *out, uint32_t rows, uint32_t src_rows, uint32_t cols, void *stream);
int launch_bias_add(const float *x, const float *bias, float *out, uint32_t rows, uint32_t cols, void *stream);
int launch_glu(const float *gate, const float *up, void *out, bool out_bf16, size_t len, const Glu &act, void *stream);
int launch_cast(const float *x, __nv_bfloat16 *out, size_t len, void *stream);
int launch_scaled_sum(const float *a, const float *b, float *out, size_t len, float sa, float sb, void *stream);

// Norm behind a sublayer: y = sa * a + sb * b (b null: sa * a), out = addend + unit_rms(y) * (offset + weight);
// copy: a second, bf16 output or null.
struct ResidualNorm {
    const float *a, *b, *weight, *addend;
    float *out;
    __nv_bfloat16 *copy;
    uint32_t rows, cols;
    float sa, sb, eps, offset;
};
int launch_residual_norm(const ResidualNorm &a, void *stream);

// h = norm_weight ? unit_rms(x) * (offset + norm_weight) : x;  out[s][r] = h[r] + (h[r-1] - h[r]) * mu[s],
// slots `slot_stride` elements apart.  state is [2, width]: row 0 is the h before row 0, row 1 receives
// the last h (committed to row 0 by the recurrence that follows, so that no CTA reads what another writes).
struct TokenShift {
    const float *x, *norm_weight;
    float eps, offset;
    const float *mu[kMaxShifts];
    uint32_t slots, rows, width;
    float *state;
    void *out;
    bool out_bf16;
    size_t slot_stride;
};
int launch_token_shift(const TokenShift &a, void *stream);

// Per-head norm and output gate: out = unit_rms(o head) * weight * act(gate); no weight: out = o * act(gate).
// shared: one weight of a head's size for all heads.
struct HeadGate {
    const float *weight, *gate;
    void *out;
    bool out_bf16, silu, shared;
    float eps;
};
int launch_head_gate(const float *o, const HeadGate &hg, uint32_t rows, uint32_t heads, uint32_t dim, void *stream);

// Decay of every key channel from a low-rank projection: low [rows, rank], w2 bf16 [channels, rank], w0 [channels].
//   inv_tau == 0:  exp(-exp(tanh(low) . w2^T + w0))
//   inv_tau  > 0:  sigmoid(low . w2^T + w0)^inv_tau
struct Decay {
    const float *low, *w0;
    const void *w2;
    float *out;                            // [rows, channels]
    uint32_t rows, channels, rank;
    float inv_tau;
};
int launch_decay(const Decay &a, void *stream);
__device__ __forceinline__ float log_sigmoid(float z) { return z < 0.f ? z - log1pf(expf(z)) : -log1pf(expf(-z)); }
__device__ __forceinline__ float decay_input(float low, float inv_tau) { return inv_tau == 0.f ? tanhf(low) : low; }
__device__ __forceinline__ float decay_value(float z, float inv_tau)
{
    if (inv_tau == 0.f) return expf(-expf(z));
    return expf((fminf(z, 0.f) - logf(1.0f + expf(-fabsf(z)))) * inv_tau);       // close to 1 only the absolute error of the logarithm counts
}

// Recurrences with a decay per key channel.  q, k, d.out [rows, heads * dim], v, o [rows, heads * vdim].
//   u set (RWKV-style):        o = (S + diag(u) k v^T)^T q, then S = diag(decay) S + k v^T
//   u null (gated linear):     S = diag(decay) S + k v^T, then o = S^T q * dim^-1/2
// State per head: [vdim values][pad4(dim) keys] f32; shift_state (may be null) is committed.
struct ChannelDecay {
    const float *q, *k, *v, *u;
    Decay d;
    float *o, *state, *shift_state;
    uint32_t rows, heads, dim, vdim, shift_width;
    void *workspace;                       // scan_workspace bytes, or null (long portions then run in one piece)
    bool split_products;                   // gated linear, kPrefillRows or more rows: chunks on the tensor cores (mgq_gla_chunks.cu),
                                           // whose workspace is gla_chunks_workspace bytes
    bool decay_pending;                    // d.out is not computed yet (only with that form, which computes the decay itself)
};
size_t channel_decay_state_elements(uint32_t heads, uint32_t dim, uint32_t vdim);
int launch_channel_decay_scan(const ChannelDecay &a, void *stream);
size_t gla_chunks_workspace(uint32_t max_rows, uint32_t heads, uint32_t dim, uint32_t vdim);
int launch_gla_chunks(const ChannelDecay &a, void *stream);
int launch_channel_decay_step(const ChannelDecay &a, const HeadGate &hg, void *stream);      // rows == 1: decay, recurrence, head gate in one launch

// mLSTM recurrence.  q, k [rows, heads * dim], v, o [rows, heads * vdim], gate pre-activations
// gi, gf [rows, heads].  State: per head [vdim][pad4(dim)], then n and m per head and block of columns.
struct Mlstm {
    const float *q, *k, *v, *gi, *gf;
    float *o, *state;
    uint32_t rows, heads, dim, vdim;
    float cap;
    void *workspace;                       // as in ChannelDecay
};
size_t scan_workspace(uint32_t max_rows, uint32_t heads, uint32_t dim, uint32_t vdim);
size_t mlstm_state_elements(uint32_t heads, uint32_t dim, uint32_t vdim);
int launch_mlstm_scan(const Mlstm &a, void *stream);
int launch_mlstm_step(const Mlstm &a, const HeadGate &hg, void *stream);

// Latent attention.  The cache is a ring of `slots` rows of rank + rot_dim elements (position p lives
// in row p % slots); freq has rot_dim / 2 entries.
struct LatentCache {
    const float *down, *weight, *freq;     // down [rows, rank + rot_dim]
    void *cache;
    bool cache_bf16;
    const uint32_t *pos;                   // position of row 0
    uint32_t rows, rank, rot_dim, slots;
    float eps;
};
int launch_latent_cache_write(const LatentCache &a, void *stream);

struct LatentAttention {
    const float *q, *freq;                 // q [rows, heads * (dim + rot_dim)]
    const void *cache, *uk, *uv;           // uk [heads * dim, rank], uv [heads * vdim, rank], bf16
    bool cache_bf16;
    const uint32_t *pos;
    float *o;                              // [rows, heads * vdim]; unused when gated
    uint32_t rows, heads, dim, rot_dim, vdim, rank, slots, window;
    float scale;
    void *workspace;
    const HeadGate *gate;                  // no weight: gate fused into the output; null: plain o
};
size_t latent_attention_workspace(uint32_t max_rows, uint32_t heads, uint32_t dim, uint32_t rot_dim, uint32_t vdim, uint32_t rank, uint32_t slots,
                                  uint32_t window, bool cache_bf16);
int launch_latent_attention(const LatentAttention &a, void *stream);
// Many rows, bf16 cache, sizes in multiples of 8 (mgq_prefill_attention.cu): keys and values are expanded
// from the latents once per step and the softmax runs tile by tile on the tensor cores.
bool latent_prefill_eligible(uint32_t dim, uint32_t rot_dim, uint32_t vdim, uint32_t rank, bool cache_bf16);
size_t latent_prefill_workspace(uint32_t heads, uint32_t dim, uint32_t rot_dim, uint32_t vdim, uint32_t slots);
int launch_latent_prefill(const LatentAttention &a, void *stream);

// Causal softmax attention over caches of `slots` positions, keys [slots, kv_heads * dim] and values
// [slots, kv_heads * vdim], f32 or f16; query head h reads key / value head h / (heads / kv_heads).
// q is [rows, heads * dim] f32, the row r at position pos + r.
struct Attention {
    const float *q;
    const void *keys, *values;
    bool half;
    const uint32_t *pos;
    float *o;                              // [rows, heads * vdim]; unused when gated
    uint32_t rows, heads, kv_heads, dim, vdim, slots;
    float scale;
    void *workspace;
    const HeadGate *gate;                  // no weight: gate fused into the output; null: plain o
};
size_t attention_workspace(uint32_t max_rows, uint32_t heads, uint32_t kv_heads, uint32_t dim, uint32_t vdim, uint32_t slots, bool half);
int launch_attention(const Attention &a, void *stream);
bool attention_prefill_eligible(const Attention &a);
int launch_attention_prefill(const Attention &a, void *stream);          // mgq_prefill_attention.cu

// out[r] = x[r] * (1 + coef * ln(floor((p + 1) / every) + 1)) at position p = pos + r
int launch_query_temperature(const float *x, const uint32_t *pos, float *out, uint32_t rows, uint32_t cols, float coef, float every, void *stream);
// cache[pos + r] = x[r]; rows beyond the cache are dropped
int launch_cache_append(const float *x, void *cache, bool half, const uint32_t *pos, uint32_t rows, uint32_t cols, uint32_t slots, void *stream);

// What stands between the projections and the attention, in one launch: query and key norm over all heads,
// query temperature, keys and values into their caches.
struct AttentionInputs {
    const float *q, *k, *v, *q_weight, *k_weight;
    const uint32_t *pos;
    float *q_out;
    void *keys, *values;
    bool half;
    uint32_t rows, q_cols, k_cols, v_cols, slots;
    float q_eps, k_eps, q_offset, k_offset, coef, every;
};
int launch_attention_inputs(const AttentionInputs &a, void *stream);

}  // namespace mgq
