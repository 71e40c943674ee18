// Matrix products in true fp32 (no tensor cores, no reduced-precision mode): out[b] = act(X[b] * W[b]^T + bias) for a batch of
// independent products. Serves the 32-bit mode of the serving programs, where exactness matters and speed does not.
#include "common.cuh"
#include "sm100_ptx.cuh"

namespace ovb {

namespace {

constexpr int FT = 64, FK = 16;   // tile of tokens and of outputs, depth of a step

struct GemmF32Params {
    const float* x;
    const float* w;
    const float* bias;
    float* out;
    long long sx, sw, sb, so;     // elements between the batch members' operands
    int T, N, K, ldx, ldw, ldo, act;
    float limit;                  // OVB_ACT_SOFTCAP
};

__global__ void __launch_bounds__(256) gemm_f32_kernel(GemmF32Params p) {
    pdl_enter();
    __shared__ float sx[FK][FT + 4], sw[FK][FT + 4];
    const int t0 = blockIdx.y * FT, n0 = blockIdx.x * FT;
    const float* x = p.x + blockIdx.z * p.sx;
    const float* w = p.w + blockIdx.z * p.sw;
    float* out = p.out + blockIdx.z * p.so;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < p.K; k0 += FK) {
        for (int i = threadIdx.x; i < FT * FK; i += 256) {
            const int r = i / FK, k = i % FK;
            sx[k][r] = (t0 + r < p.T && k0 + k < p.K) ? x[(size_t)(t0 + r) * p.ldx + k0 + k] : 0.f;
            sw[k][r] = (n0 + r < p.N && k0 + k < p.K) ? w[(size_t)(n0 + r) * p.ldw + k0 + k] : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < FK; ++k) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                a[i] = sx[k][ty * 4 + i];
                b[i] = sw[k][tx * 4 + i];
            }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int t = t0 + ty * 4 + i, n = n0 + tx * 4 + j;
            if (t >= p.T || n >= p.N) continue;
            float v = acc[i][j];
            if (p.bias) v += p.bias[blockIdx.z * p.sb + n];
            if (p.act == OVB_ACT_GELU_TANH) v = 0.5f * v * (1.f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v)));
            else if (p.act == OVB_ACT_SILU) v = v / (1.f + expf(-v));
            else if (p.act == OVB_ACT_RELU) v = fmaxf(v, 0.f);
            else if (p.act == OVB_ACT_RELU2) v = fmaxf(v, 0.f) * v;
            else if (p.act == OVB_ACT_SOFTCAP) v = p.limit * tanhf(v / p.limit);
            out[(size_t)t * p.ldo + n] = v;
        }
}

}  // namespace

}  // namespace ovb

extern "C" int ovb_gemm_f32(const float* x, const float* w, const float* bias, float* out, int batch, long long sx, long long sw, long long sb, long long so,
                            int T, int N, int K, int ldx, int ldw, int ldo, int act, float act_limit, ovb_stream_t stream) {
    using namespace ovb;
    OVB_REQUIRE(x && w && out && batch > 0 && T > 0 && N > 0 && K > 0 && batch <= 65535, "ovb_gemm_f32: bad arguments");
    OVB_REQUIRE(ceil_div(T, FT) <= 65535, "ovb_gemm_f32: %d rows are too many", T);
    OVB_REQUIRE(act == OVB_ACT_NONE || act == OVB_ACT_GELU_TANH || act == OVB_ACT_SILU || act == OVB_ACT_RELU || act == OVB_ACT_RELU2 ||
                    (act == OVB_ACT_SOFTCAP && act_limit > 0.f), "ovb_gemm_f32: activation %d is not served", act);
    GemmF32Params p = {x, w, bias, out, sx, sw, sb, so, T, N, K, ldx, ldw, ldo, act, act_limit};
    OVB_CHECK_CUDA(launch_pdl(gemm_f32_kernel, dim3(ceil_div(N, FT), ceil_div(T, FT), batch), dim3(256), 0, (cudaStream_t)stream, p));
    return 0;
}
