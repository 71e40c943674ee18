// Short causal convolution over time, one filter per channel: y[pos] = sum_j w[j] * u[pos - (taps - 1) + j], zeros before position 0.
//
// The inputs u are columns of a projection. Those of earlier steps come from a ring per request slot, [taps, cols] fp32, that holds
// the input of position p in row p % taps. The taps - 1 rows that a token reads are never the row of the token itself, so a decode step
// reads and writes the ring in one kernel; a step with longer pieces brings it up to date behind its last reader
// (ovb_conv_ring_update). What a slot's earlier owner left is never read: a sequence only looks at positions that it has written.
#pragma once
#include "store_types.cuh"

namespace ovb {

struct ShortConv {
    const float* w;      // [taps, cols]
    float* ring;         // [slots, taps, cols]
    int taps, cols;
};

// Input of the convolution `back` positions before token t (position pos) of a sequence whose tokens of this step begin at row `begin`;
// x: column of the projection, ring: the same channel of the slot's ring.
template <class E>
__device__ __forceinline__ float conv_input(const E* x, int ldx, const float* ring, const ShortConv& cv, int t, int begin, int pos, int back) {
    if (t - back >= begin) return ld_f32(x + (size_t)(t - back) * ldx);
    if (pos - back < 0) return 0.f;
    return ring[(size_t)((pos - back) % cv.taps) * cv.cols];
}
template <class E>
__device__ __forceinline__ float4 conv_input4(const E* x, int ldx, const float* ring, const ShortConv& cv, int t, int begin, int pos, int back) {
    if (t - back >= begin) return ld4_f32(x + (size_t)(t - back) * ldx);
    if (pos - back < 0) return make_float4(0.f, 0.f, 0.f, 0.f);
    return ld4_f32(ring + (size_t)((pos - back) % cv.taps) * cv.cols);
}

__device__ __forceinline__ float4 fma4(float4 a, float4 b, float4 c) {
    return make_float4(fmaf(a.x, b.x, c.x), fmaf(a.y, b.y, c.y), fmaf(a.z, b.z, c.z), fmaf(a.w, b.w, c.w));
}

}  // namespace ovb
