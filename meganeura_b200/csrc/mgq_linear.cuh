// A group of linear layers that one launch computes (mgq_linear.cu, mgq_linear_tc.cu).
#pragma once
#include "mgq_launch.cuh"

namespace mgq {

constexpr uint32_t kMaxSegments = 12;

struct LinearSegment {
    const void *a;                // [m, k] activations, f32 or bf16
    const void *w, *w2;           // [n, k] bf16; w2: the up projection of a GLU pair (w is the gate)
    const float *bias, *bias2;    // [n] or null (a GLU pair has both or none)
    const float *addend;          // [m, n] f32 or null
    void *out;                    // [m, n] f32, or bf16 when the group says so
    uint32_t n, k;
};

struct LinearGroup {
    LinearSegment seg[kMaxSegments];
    uint32_t count, m;
    uint32_t a_bf16, glu;
    uint32_t out_bf16;            // GLU only
    uint32_t out_f16;             // tcgen05 path without an addend: f16, clamped to its range
    uint32_t lda;                 // elements between rows of a; 0: k (tcgen05 path only)
    const uint32_t *live;         // tcgen05 path: only rows below *live + live_add are wanted; null: all
    uint32_t live_add;
    Glu act;                      // GLU
};

int launch_linear_group(const LinearGroup &g, void *stream);
// tcgen05 path: bf16 activations, k % 8 == 0, 16-byte aligned operands.
int launch_linear_tc(const LinearGroup &g, void *stream);

}  // namespace mgq
