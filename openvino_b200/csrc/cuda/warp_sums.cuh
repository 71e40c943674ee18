// Sums of several per-lane values over a warp with few shuffles.
#pragma once

namespace ovb {

// Sums four per-lane values over the warp with 6 shuffles instead of 20: after each exchange a lane keeps only the values
// its half is responsible for. The total of v0 ends in lanes 0-7, v1 in 16-23, v2 in 8-15, v3 in 24-31.
__device__ __forceinline__ float rec_reduce4(float v0, float v1, float v2, float v3, int lane) {
    const bool up16 = lane & 16, up8 = lane & 8;
    float a = (up16 ? v1 : v0) + __shfl_xor_sync(0xffffffffu, up16 ? v0 : v1, 16);
    float b = (up16 ? v3 : v2) + __shfl_xor_sync(0xffffffffu, up16 ? v2 : v3, 16);
    float c = (up8 ? b : a) + __shfl_xor_sync(0xffffffffu, up8 ? a : b, 8);
    c += __shfl_xor_sync(0xffffffffu, c, 4);
    c += __shfl_xor_sync(0xffffffffu, c, 2);
    c += __shfl_xor_sync(0xffffffffu, c, 1);
    return c;
}
// Lane that holds the total of value r after rec_reduce4, and the value index a lane holds
__device__ __forceinline__ int rec_owner_lane(int r) { return ((r & 1) << 4) | ((r >> 1) << 3); }
__device__ __forceinline__ int rec_owned_value(int lane) { return ((lane >> 4) & 1) | (((lane >> 3) & 1) << 1); }

// Sums eight per-lane values over the warp with 9 shuffles. The total of value r ends in the four lanes whose bits 4, 3, 2
// spell r & 1, (r >> 1) & 1, (r >> 2) & 1.
__device__ __forceinline__ float rec_reduce8(const float (&v)[8], int lane) {
    const bool up16 = lane & 16, up8 = lane & 8, up4 = lane & 4;
    float a[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) a[i] = (up16 ? v[2 * i + 1] : v[2 * i]) + __shfl_xor_sync(0xffffffffu, up16 ? v[2 * i] : v[2 * i + 1], 16);
    float b0 = (up8 ? a[1] : a[0]) + __shfl_xor_sync(0xffffffffu, up8 ? a[0] : a[1], 8);
    float b1 = (up8 ? a[3] : a[2]) + __shfl_xor_sync(0xffffffffu, up8 ? a[2] : a[3], 8);
    float c = (up4 ? b1 : b0) + __shfl_xor_sync(0xffffffffu, up4 ? b0 : b1, 4);
    c += __shfl_xor_sync(0xffffffffu, c, 2);
    c += __shfl_xor_sync(0xffffffffu, c, 1);
    return c;
}
__device__ __forceinline__ int rec_owned_value8(int lane) { return ((lane >> 4) & 1) | (((lane >> 3) & 1) << 1) | (((lane >> 2) & 1) << 2); }

}  // namespace ovb
