// Short causal convolution over time, one filter per channel: y[pos] = sum_j w[j] * u[pos - (taps - 1) + j], zeros before position 0.
//
// The inputs u are columns of a projection. Those of earlier steps come from a ring per request slot, [taps, cols] fp32, that holds
// the input of position p in row p % taps. The taps - 1 rows that a token reads are never the row of the token itself, so a decode step
// reads and writes the ring in one kernel; a step with longer pieces brings it up to date behind its last reader
// (update_conv_ring). What a slot's earlier owner left is never read: a sequence only looks at positions that it has written.
#pragma once
#include "sm100_ptx.cuh"
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

// Inputs of a step's last taps - 1 positions of every sequence -> rings.
template <class E>
__global__ void __launch_bounds__(128) conv_ring_update_kernel(const E* __restrict__ proj, float* __restrict__ ring, const int* __restrict__ begins,
                                                               const int* __restrict__ past_lens, const int* __restrict__ slots, int cols, int taps, int ldp) {
    pdl_enter();
    const int b = blockIdx.y, c = blockIdx.x * 128 + threadIdx.x;
    if (c >= cols) return;
    const int begin = begins[b], end = begins[b + 1], past = past_lens[b];
    float* mine = ring + (size_t)slots[b] * taps * cols + c;
    for (int t = max(begin, end - (taps - 1)); t < end; ++t) mine[(size_t)((past + t - begin) % taps) * cols] = ld_f32(proj + (size_t)t * ldp + c);
}

template <class E>
inline int update_conv_ring(const void* proj, int ldp, const ShortConv& cv, const int* begins, const int* past_lens, const int* slots, int B, cudaStream_t stream) {
    if (cv.taps <= 1) return 0;
    OVB_CHECK_CUDA(launch_pdl(conv_ring_update_kernel<E>, dim3(ceil_div(cv.cols, 128), B), dim3(128), 0, stream, reinterpret_cast<const E*>(proj), cv.ring, begins,
                              past_lens, slots, cv.cols, cv.taps, ldp));
    return 0;
}

__device__ __forceinline__ float4 fma4(float4 a, float4 b, float4 c) {
    return make_float4(fmaf(a.x, b.x, c.x), fmaf(a.y, b.y, c.y), fmaf(a.z, b.z, c.z), fmaf(a.w, b.w, c.w));
}

}  // namespace ovb
