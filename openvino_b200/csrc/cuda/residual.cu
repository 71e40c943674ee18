// A residual stream kept in fp32: token embedding, "sum, then norm" (one or two norms of the same sum) and the clamped gated MLP
// activation.
//
// The stream h is [rows, ldh] fp32; x is the copy of it in the storage type of the matrix products (bf16, or none when the
// products themselves run in fp32 and read h). Row pitches are multiples of four elements; columns between the width and
// the next multiple of four read as zeros and are written as zeros.
#include "sm100_ptx.cuh"
#include "store_types.cuh"

namespace ovb {

namespace {

constexpr int kNormThreads = 256;

template <class E>
__global__ void stream_embed_kernel(const int* __restrict__ ids, const E* __restrict__ table, float* __restrict__ h, E* __restrict__ x, int cols,
                                    int vocab, int ldt, int ldh, int ldx) {
    pdl_enter();
    const int row = blockIdx.x;
    int id = ids[row];
    if ((unsigned)id >= (unsigned)vocab) id = 0;
    const E* src = table + (size_t)id * ldt;
    const int nvec = (cols % 4 == 0 && ldt % 4 == 0) ? cols / 4 : 0;
    for (int k = threadIdx.x; k < nvec; k += blockDim.x) {
        const float4 v = ld4_f32(src + k * 4);
        st4_f32(h + (size_t)row * ldh + k * 4, v);
        if (x) st4_f32(x + (size_t)row * ldx + k * 4, v);
    }
    for (int c = nvec * 4 + threadIdx.x; c < cols; c += blockDim.x) {
        const float v = ld_f32(src + c);
        h[(size_t)row * ldh + c] = v;
        if (x) st_f32(x + (size_t)row * ldx + c, v);
    }
}

// s = alpha * h[src row] (+ y[src row]);  out = s / sqrt(mean(s^2) + eps) * (w_offset + w), for up to two weights.  One CTA per row,
// the row stays in registers.
template <class E, int MAXV>
__global__ void __launch_bounds__(kNormThreads) sum_rmsnorm_kernel(ovb_sum_rmsnorm_args p) {
    pdl_enter();
    __shared__ float red[kNormThreads / 32];
    const int row = blockIdx.x, src = p.row_idx ? p.row_idx[row] : row;
    const int nvec = (p.cols + 3) / 4;
    float4 v[MAXV];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < MAXV; ++i) {
        const int k = threadIdx.x + i * kNormThreads;
        v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (k < nvec) {
            const float4 a = ld4_f32(p.h + (size_t)src * p.ldh + k * 4);
            v[i] = make_float4(p.alpha * a.x, p.alpha * a.y, p.alpha * a.z, p.alpha * a.w);
            if (p.y) {
                const float4 b = ld4_f32(p.y + (size_t)src * p.ldy + k * 4);
                v[i].x += b.x; v[i].y += b.y; v[i].z += b.z; v[i].w += b.w;
            }
            ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
        }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int i = 0; i < kNormThreads / 32; ++i) tot += red[i];
    const float inv = 1.f / sqrtf(tot / (float)p.cols + p.eps);
    E* x_out = reinterpret_cast<E*>(p.x_out);
    E* x2_out = reinterpret_cast<E*>(p.x2_out);
#pragma unroll
    for (int i = 0; i < MAXV; ++i) {
        const int k = threadIdx.x + i * kNormThreads;
        if (k < nvec) {
            if (p.s_out) st4_f32(p.s_out + (size_t)row * p.lds + k * 4, v[i]);
            auto weighted = [&](const float* w) {
                const float4 g = ld4_f32(w + k * 4);
                return make_float4(v[i].x * inv * (p.w_offset + g.x), v[i].y * inv * (p.w_offset + g.y), v[i].z * inv * (p.w_offset + g.z),
                                   v[i].w * inv * (p.w_offset + g.w));
            };
            const float4 o = weighted(p.w);
            if (p.h_out) st4_f32(p.h_out + (size_t)row * p.ldho + k * 4, o);
            if (x_out) st4_f32(x_out + (size_t)row * p.ldx + k * 4, o);
            if (x2_out) st4_f32(x2_out + (size_t)row * p.ldx2 + k * 4, weighted(p.w2));
        }
    }
}

// g = min(gate, limit), u = clamp(up, -limit, limit);  out = g * sigmoid(slope * g) * (u + shift).
template <class E>
__global__ void glu_limited_kernel(const E* __restrict__ gu, E* __restrict__ out, int rows, int F, int up_off, int ldg, int ldo, float limit, float slope,
                                   float shift) {
    pdl_enter();
    const size_t n = (size_t)rows * F;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
        const size_t r = i / F;
        const int c = (int)(i % F);
        const float g = fminf(ld_f32(gu + r * ldg + c), limit);
        const float u = fminf(fmaxf(ld_f32(gu + r * ldg + up_off + c), -limit), limit);
        st_f32(out + r * ldo + c, g / (1.f + expf(-slope * g)) * (u + shift));
    }
}

template <class E>
int launch_sum_rmsnorm(const ovb_sum_rmsnorm_args& a, cudaStream_t stream) {
    auto go = [&](auto kern) -> int {
        OVB_CHECK_CUDA(launch_pdl(kern, dim3(a.rows), dim3(kNormThreads), 0, stream, a));
        return 0;
    };
    const int per = ceil_div(ceil_div(a.cols, 4), kNormThreads);
    if (per <= 1) return go(sum_rmsnorm_kernel<E, 1>);
    if (per <= 2) return go(sum_rmsnorm_kernel<E, 2>);
    if (per <= 4) return go(sum_rmsnorm_kernel<E, 4>);
    if (per <= 8) return go(sum_rmsnorm_kernel<E, 8>);
    if (per <= 16) return go(sum_rmsnorm_kernel<E, 16>);
    set_error("ovb_sum_rmsnorm: width %d above %d", a.cols, 16 * 4 * kNormThreads);
    return ERR_UNSUPPORTED;
}

}  // namespace

}  // namespace ovb

extern "C" {
using namespace ovb;

int ovb_stream_embed(const int* ids, const void* table, float* h, void* x, int rows, int cols, int vocab, int ldt, int ldh, int ldx, int dtype,
                     ovb_stream_t stream) {
    OVB_REQUIRE(ids && table && h && rows > 0 && cols > 0 && vocab > 0 && ldh % 4 == 0 && ldx % 4 == 0, "ovb_stream_embed: bad arguments");
    return dispatch_store(dtype, "ovb_stream_embed", [&](auto e) -> int {
        using E = decltype(e);
        OVB_CHECK_CUDA(launch_pdl(stream_embed_kernel<E>, dim3(rows), dim3(256), 0, (cudaStream_t)stream, ids, (const E*)table, h, (E*)x, cols, vocab, ldt,
                                  ldh, ldx));
        return 0;
    });
}

int ovb_sum_rmsnorm(const ovb_sum_rmsnorm_args* a, ovb_stream_t stream) {
    OVB_REQUIRE(a && a->h && a->w && (a->h_out || a->x_out) && a->rows > 0 && a->cols > 0 && (a->x2_out == nullptr || a->w2), "ovb_sum_rmsnorm: bad arguments");
    OVB_REQUIRE(a->ldh % 4 == 0 && a->ldy % 4 == 0 && a->ldho % 4 == 0 && a->lds % 4 == 0 && a->ldx % 4 == 0 && a->ldx2 % 4 == 0,
                "ovb_sum_rmsnorm: row pitches must be multiples of 4 elements");
    return dispatch_store(a->dtype, "ovb_sum_rmsnorm", [&](auto e) -> int {
        using E = decltype(e);
        return launch_sum_rmsnorm<E>(*a, (cudaStream_t)stream);
    });
}

int ovb_glu_limited(const void* gu, void* out, int rows, int F, int up_off, int ldg, int ldo, float limit, float slope, float shift, int dtype,
                    ovb_stream_t stream) {
    OVB_REQUIRE(gu && out && rows > 0 && F > 0, "ovb_glu_limited: bad arguments");
    return dispatch_store(dtype, "ovb_glu_limited", [&](auto e) -> int {
        using E = decltype(e);
        const size_t n = (size_t)rows * F;
        const int grid = (int)((n + 255) / 256 < 4736 ? (n + 255) / 256 : 4736);
        OVB_CHECK_CUDA(launch_pdl(glu_limited_kernel<E>, dim3(grid), dim3(256), 0, (cudaStream_t)stream, (const E*)gu, (E*)out, rows, F, up_off, ldg, ldo,
                                  limit, slope, shift));
        return 0;
    });
}

}  // extern "C"
