// Operators of decoders with recurrent and latent-attention mixers (mgq_mixer_ops.cu,
// mgq_latent_attention.cu).  All pointers are device pointers; activations are f32 unless an
// argument says bf16; `rows` consecutive tokens of one sequence.
#pragma once
#include "mgq_launch.cuh"

namespace mgq {

constexpr int kMaxShifts = 8;
constexpr uint32_t kMaxStateDim = 256;         // key dimensions of a recurrent head

// out[r] = table[ids[r]] * scale
int launch_embedding_scaled(const uint32_t *ids, const void *table, bool table_bf16, float *out, uint32_t rows, uint32_t width, uint32_t vocab,
                            float scale, void *stream);
// out[r] = unit_rms(x[index ? index[r] : r]) * (offset + weight)
int launch_norm(const float *x, const float *weight, const uint32_t *index, void *out, bool out_bf16, uint32_t rows, uint32_t src_rows,
                uint32_t cols, float eps, float offset, void *stream);
int launch_pick_rows(const float *x, const uint32_t *index, float *out, uint32_t rows, uint32_t src_rows, uint32_t cols, void *stream);
int launch_bias_add(const float *x, const float *bias, float *out, uint32_t rows, uint32_t cols, void *stream);
int launch_clamped_glu(const float *gate, const float *up, void *out, bool out_bf16, size_t len, float limit, float alpha, void *stream);

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
struct HeadGate {
    const float *weight, *gate;
    void *out;
    bool out_bf16, silu;
    float eps;
};
int launch_head_gate(const float *o, const HeadGate &hg, uint32_t rows, uint32_t heads, uint32_t dim, void *stream);

// RWKV-style recurrence.  r, k, v [rows, heads * dim]; decay = exp(-exp(tanh(low) . w2^T + w0)) with
// low [rows, rank], w2 bf16 [heads * dim, rank].  `decay` and `o` are [rows, heads * dim].
// State per head: [dim values][pad4(dim) keys] f32; shift_state (may be null) is committed.
struct Wkv {
    const float *r, *k, *v, *low, *w0, *u;
    const void *w2;
    float *decay, *o, *state, *shift_state;
    uint32_t rows, heads, dim, rank, shift_width;
    void *workspace;                       // scan_workspace bytes, or null (long portions then run in one piece)
};
size_t wkv_state_elements(uint32_t heads, uint32_t dim);
int launch_decay(const Wkv &a, void *stream);
int launch_wkv_scan(const Wkv &a, void *stream);
int launch_wkv_step(const Wkv &a, const HeadGate &hg, void *stream);      // rows == 1: decay, recurrence, head gate in one launch

// mLSTM recurrence.  q, k [rows, heads * dim], v, o [rows, heads * vdim], gate pre-activations
// gi, gf [rows, heads].  State: per head [vdim][pad4(dim)], then n and m per head and block of columns.
struct Mlstm {
    const float *q, *k, *v, *gi, *gf;
    float *o, *state;
    uint32_t rows, heads, dim, vdim;
    float cap;
    void *workspace;                       // as in Wkv
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
// Many rows, bf16 cache, sizes in multiples of 8 (mgq_latent_prefill.cu): keys and values are expanded
// from the latents once per step and the softmax runs tile by tile on the tensor cores.
constexpr uint32_t kPrefillRows = 64;      // fewer rows take the absorbed form
bool latent_prefill_eligible(uint32_t dim, uint32_t rot_dim, uint32_t vdim, uint32_t rank, bool cache_bf16);
size_t latent_prefill_workspace(uint32_t heads, uint32_t dim, uint32_t rot_dim, uint32_t vdim, uint32_t slots);
int launch_latent_prefill(const LatentAttention &a, void *stream);

}  // namespace mgq
