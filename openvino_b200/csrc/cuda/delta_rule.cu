// Gated delta rule with a decay per key channel, fused with everything between its projections and the output projection: short
// convolutions, silu, unit norms, decays, step sizes, the recurrence, the norm of its read-out and the output gate.
//
// The state S [dk, dv] of a head stays in registers for the whole piece of a sequence that a step brings and touches memory twice. Its
// columns are independent: lane l of a consumer warp holds CPT columns (column group l % 8) at RL rows (row group l / 8), so that the dot
// products over the rows are sums within a lane plus two shuffles, and no barrier stands in a token's chain
//
//     S <- g S;  m = S^T k;  o = S^T q;  u = beta (v - m);  S <- S + k u^T;  o += (k . q) u
//
// (the read-out after the update, written with the dot product k . q so that both sums run side by side). Rows are taken two at a time
// with the packed fp32 instructions of sm_100.
//
// One CTA works on (sequence, head, part of the columns). Consumer warps run the recurrence over a stage of CHUNK tokens in shared
// memory; producer warps meanwhile prepare the next stage (convolution, silu, norms, decays: one warp per token) and finish the previous
// one (norm of the read-out, gate, store). When there are too few (sequence, head) pairs to fill the machine, a cluster of CTAs shares a
// head's columns and reads each other's read-outs through distributed shared memory for the norm.
#include <cooperative_groups.h>

#include <atomic>

#include "common.cuh"
#include "short_conv.cuh"
#include "sm100_ptx.cuh"
#include "store_types.cuh"

namespace ovb {

namespace {

namespace cg = cooperative_groups;

using f32x2 = unsigned long long;      // two packed floats

__device__ __forceinline__ f32x2 pack2(float lo, float hi) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ float2 unpack2(f32x2 v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
    f32x2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ f32x2 add2(f32x2 a, f32x2 b) {
    f32x2 r;
    asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}

__device__ __forceinline__ float delta_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
// Full-precision and fast forms: the 32-bit mode takes the first.
template <class E>
struct Fn;
template <>
struct Fn<float> {
    static __device__ __forceinline__ float sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
    static __device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
};
template <>
struct Fn<__nv_bfloat16> {
    static __device__ __forceinline__ float sigmoid(float z) { return __fdividef(1.f, 1.f + __expf(-z)); }
    static __device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + __logf(1.f + __expf(-fabsf(z))); }
};

struct DeltaShape {
    int parts;               // CTAs that share a head's columns (a cluster)
    int cols;                // columns per CTA, a multiple of 8 CPT (the last part may reach past dv)
    int consumers;           // warps that run the recurrence: cols / (8 CPT)
    int chunk;               // tokens per stage
};

// Floats of one stage: K, Q, G [chunk][DP], V [chunk][cols], beta and k . q [chunk] (padded to whole 16-byte pieces).
__host__ __device__ inline int stage_floats(int dp, int cols, int chunk) { return chunk * (3 * dp + cols) + (2 * chunk + 3) / 4 * 4; }

template <class E, int RL, int CPT>
__global__ void __launch_bounds__(384, 1) channel_delta_kernel(ovb_delta_args p, DeltaShape s) {
    constexpr int DP = RL * 4;                     // rows, zero behind p.dk
    extern __shared__ __align__(16) float smem[];
    const int stage_len = stage_floats(DP, s.cols, s.chunk);
    float* y_buf = smem + 2 * stage_len;           // [2][chunk][cols] read-outs
    float* s_conv = y_buf + 2 * s.chunk * s.cols;  // [taps][2 DP + cols] filters of the head's q, k and of this CTA's v columns
    const int conv_len = 2 * DP + s.cols;
    float* s_bias = s_conv + p.taps * conv_len;    // [DP]
    float* s_norm = s_bias + DP;                   // [cols]

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = blockDim.x >> 5;
    const int part = blockIdx.x % s.parts, h = blockIdx.x / s.parts, b = blockIdx.y;
    const int c0 = part * s.cols, kvh = h / (p.H / p.G);
    const bool consumer = warp < s.consumers;
    cg::cluster_group cluster = cg::this_cluster();
    auto barrier = [&]() {
        if (s.parts > 1) cluster.sync();
        else __syncthreads();
    };

    // constants of the head (weights: no earlier kernel of the stream writes them)
    for (int i = threadIdx.x; i < p.taps * conv_len; i += blockDim.x) {
        const int j = i / conv_len, c = i % conv_len;
        const bool is_v = c >= 2 * DP;
        const int r = is_v ? c0 + c - 2 * DP : c % DP;                       // column within the head
        const int col = is_v ? p.v_off + h * p.dv + r : (c < DP ? 0 : p.k_off) + kvh * p.dk + r;
        s_conv[i] = r < (is_v ? p.dv : p.dk) ? p.conv_w[(size_t)j * p.conv_cols + col] : 0.f;
    }
    for (int i = threadIdx.x; i < DP; i += blockDim.x) s_bias[i] = i < p.dk ? p.dt_bias[(size_t)h * p.dk + i] : 0.f;
    for (int i = threadIdx.x; i < s.cols; i += blockDim.x) s_norm[i] = c0 + i < p.dv ? p.norm[c0 + i] : 0.f;
    const float decay_a = p.decay_a[h];
    pdl_enter();

    const int begin = p.subsequence_begins[b], len = p.subsequence_begins[b + 1] - begin, past = p.past_lens[b], slot = p.slots[b];
    const E* proj = reinterpret_cast<const E*>(p.proj);
    const ShortConv cv = {p.conv_w, p.conv_ring, p.taps, p.conv_cols};
    float* ring = p.conv_ring + (size_t)slot * p.taps * p.conv_cols;
    const bool single = p.max_q_len == 1 && p.taps > 1;       // this kernel keeps the ring up to date
    const bool ring_owner = single && part == 0 && h % (p.H / p.G) == 0;

    // convolution and silu of four columns of token t
    auto conv_silu = [&](int col, const float* w, int t) {
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int j = 0; j < p.taps; ++j)
            acc = fma4(ld4_f32(w + j * conv_len), conv_input4(proj + col, p.ldp, ring + col, cv, t, begin, past + t - begin, p.taps - 1 - j), acc);
        return make_float4(acc.x * Fn<E>::sigmoid(acc.x), acc.y * Fn<E>::sigmoid(acc.y), acc.z * Fn<E>::sigmoid(acc.z), acc.w * Fn<E>::sigmoid(acc.w));
    };
    auto keep_input = [&](int col, int t) {
        st4_f32(ring + (size_t)((past + t - begin) % p.taps) * p.conv_cols + col, ld4_f32(proj + (size_t)t * p.ldp + col));
    };

    // one unit: the keys, queries and decays of a token (kind 0), or its values and step size (kind 1)
    auto stage_unit = [&](float* st, int tt, int kind, int t) {
        if (kind == 0) {
            constexpr int NV = (DP + 127) / 128;
            float4 q[NV], k[NV];
            float qq = 0.f, kk = 0.f, qk = 0.f;
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const int c = i * 128 + lane * 4;
                q[i] = k[i] = make_float4(0.f, 0.f, 0.f, 0.f);
                if (c < p.dk) {
                    q[i] = conv_silu(kvh * p.dk + c, s_conv + c, t);
                    k[i] = conv_silu(p.k_off + kvh * p.dk + c, s_conv + DP + c, t);
                    if (ring_owner) {
                        keep_input(kvh * p.dk + c, t);
                        keep_input(p.k_off + kvh * p.dk + c, t);
                    }
                }
                qq += q[i].x * q[i].x + q[i].y * q[i].y + q[i].z * q[i].z + q[i].w * q[i].w;
                kk += k[i].x * k[i].x + k[i].y * k[i].y + k[i].z * k[i].z + k[i].w * k[i].w;
                qk += q[i].x * k[i].x + q[i].y * k[i].y + q[i].z * k[i].z + q[i].w * k[i].w;
            }
            const float iq = p.q_scale / sqrtf(delta_sum(qq) + 1e-6f), ik = 1.f / sqrtf(delta_sum(kk) + 1e-6f);
            qk = delta_sum(qk) * iq * ik;
            const float* low = p.low + (size_t)t * p.ld_low + (size_t)h * p.dk;
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const int c = i * 128 + lane * 4;
                if (c < DP) {
                    float4 g = make_float4(1.f, 1.f, 1.f, 1.f);
                    if (c < p.dk) {
                        const float4 a = ld4_f32(low + c), bias = ld4_f32(s_bias + c);
                        g = make_float4(expf(-decay_a * Fn<E>::softplus(a.x + bias.x)), expf(-decay_a * Fn<E>::softplus(a.y + bias.y)),
                                        expf(-decay_a * Fn<E>::softplus(a.z + bias.z)), expf(-decay_a * Fn<E>::softplus(a.w + bias.w)));
                    }
                    st4_f32(st + tt * DP + c, make_float4(k[i].x * ik, k[i].y * ik, k[i].z * ik, k[i].w * ik));
                    st4_f32(st + (s.chunk + tt) * DP + c, make_float4(q[i].x * iq, q[i].y * iq, q[i].z * iq, q[i].w * iq));
                    st4_f32(st + (2 * s.chunk + tt) * DP + c, g);
                }
            }
            if (lane == 0) st[s.chunk * (3 * DP + s.cols) + s.chunk + tt] = qk;
        } else {
            for (int c = lane * 4; c < s.cols; c += 128) {
                float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
                if (c0 + c < p.dv) {
                    const int col = p.v_off + h * p.dv + c0 + c;
                    v = conv_silu(col, s_conv + 2 * DP + c, t);
                    if (single) keep_input(col, t);
                }
                st4_f32(st + 3 * s.chunk * DP + tt * s.cols + c, v);
            }
            if (lane == 0) st[s.chunk * (3 * DP + s.cols) + tt] = Fn<E>::sigmoid(ld_f32(proj + (size_t)t * p.ldp + p.b_off + h));
        }
    };
    auto stage = [&](int c, int w, int nw) {
        float* st = smem + (c & 1) * stage_len;
        const int n = min(s.chunk, len - c * s.chunk);
        for (int u = w; u < 2 * n; u += nw) stage_unit(st, u >> 1, u & 1, begin + c * s.chunk + (u >> 1));
    };
    // norm, gate and store of the read-outs of a stage; columns of the other parts of the cluster are read for the norm only
    auto finish = [&](int c, int w, int nw) {
        const int n = min(s.chunk, len - c * s.chunk);
        float* ys = y_buf + (c & 1) * s.chunk * s.cols;
        for (int tt = w; tt < n; tt += nw) {
            const size_t t = (size_t)begin + c * s.chunk + tt;
            float ss = 0.f;
            for (int col = lane * 4; col < s.parts * s.cols; col += 128) {
                const int from = col / s.cols;
                const float* row = ys + tt * s.cols + (col - from * s.cols);
                const float4 y = ld4_f32(from == part ? row : cluster.map_shared_rank(row, from));
                ss += y.x * y.x + y.y * y.y + y.z * y.z + y.w * y.w;
            }
            const float inv = 1.f / sqrtf(delta_sum(ss) / (float)p.Dv + p.eps);
            for (int col = lane * 4; col < s.cols && c0 + col < p.dv; col += 128) {
                const float4 y = ld4_f32(ys + tt * s.cols + col), w4 = ld4_f32(s_norm + col);
                const float4 g = ld4_f32(p.low + t * p.ld_low + p.gate_off + (size_t)h * p.dv + c0 + col);
                st4_f32(reinterpret_cast<E*>(p.out) + t * p.ldo + (size_t)h * p.o_head + c0 + col,
                        make_float4(y.x * inv * w4.x * Fn<E>::sigmoid(g.x), y.y * inv * w4.y * Fn<E>::sigmoid(g.y), y.z * inv * w4.z * Fn<E>::sigmoid(g.z),
                                    y.w * inv * w4.w * Fn<E>::sigmoid(g.w)));
            }
        }
    };

    // rows 16 j + 4 rg + e, columns cc .. cc + CPT - 1 of this CTA; two rows packed
    const int rg = lane >> 3, cc = warp * 8 * CPT + (lane & 7) * CPT;
    f32x2 S[RL / 2][CPT];
    float* state = p.state + ((size_t)slot * p.H + h) * p.dk * p.dv + c0 + cc;
    const bool mine = consumer && c0 + cc < p.dv;      // (dv is a multiple of 16: whole column groups)
    if (consumer) {
        const bool load = mine && past > 0;
#pragma unroll
        for (int i = 0; i < RL / 2; ++i) {
            const int r = (i >> 1) * 16 + rg * 4 + (i & 1) * 2;
            float lo[CPT], hi[CPT];
#pragma unroll
            for (int c = 0; c < CPT; ++c) lo[c] = hi[c] = 0.f;
            if (load && r < p.dk) {
                if constexpr (CPT == 2) {
                    const float2 a = *reinterpret_cast<const float2*>(state + (size_t)r * p.dv), d = *reinterpret_cast<const float2*>(state + (size_t)(r + 1) * p.dv);
                    lo[0] = a.x; lo[1] = a.y; hi[0] = d.x; hi[1] = d.y;
                } else {
                    lo[0] = state[(size_t)r * p.dv];
                    hi[0] = state[(size_t)(r + 1) * p.dv];
                }
            }
#pragma unroll
            for (int c = 0; c < CPT; ++c) S[i][c] = pack2(lo[c], hi[c]);
        }
    } else {
        stage(0, warp - s.consumers, nwarps - s.consumers);
    }
    barrier();
    const int chunks = (len + s.chunk - 1) / s.chunk;
    for (int c = 0; c < chunks; ++c) {
        if (consumer) {
            const float* st = smem + (c & 1) * stage_len;
            const float* sk = st + rg * 4;
            const float* sq = sk + s.chunk * DP;
            const float* sg = sq + s.chunk * DP;
            const float* sv = st + 3 * s.chunk * DP + cc;
            const float* sb = st + s.chunk * (3 * DP + s.cols);
            float* ys = y_buf + (c & 1) * s.chunk * s.cols + cc;
            const int n = min(s.chunk, len - c * s.chunk);
            for (int tt = 0; tt < n; ++tt) {
                f32x2 m2[CPT][2], o2[CPT][2], k2[RL / 2];
#pragma unroll
                for (int x = 0; x < CPT; ++x) m2[x][0] = m2[x][1] = o2[x][0] = o2[x][1] = 0ull;
#pragma unroll
                for (int j = 0; j < RL / 4; ++j) {
                    const ulonglong2 kk = *reinterpret_cast<const ulonglong2*>(sk + tt * DP + j * 16);
                    const ulonglong2 qq = *reinterpret_cast<const ulonglong2*>(sq + tt * DP + j * 16);
                    const ulonglong2 gg = *reinterpret_cast<const ulonglong2*>(sg + tt * DP + j * 16);
                    k2[2 * j] = kk.x;
                    k2[2 * j + 1] = kk.y;
#pragma unroll
                    for (int x = 0; x < CPT; ++x) {
                        S[2 * j][x] = mul2(S[2 * j][x], gg.x);
                        S[2 * j + 1][x] = mul2(S[2 * j + 1][x], gg.y);
                        m2[x][0] = fma2(S[2 * j][x], kk.x, m2[x][0]);
                        m2[x][1] = fma2(S[2 * j + 1][x], kk.y, m2[x][1]);
                        o2[x][0] = fma2(S[2 * j][x], qq.x, o2[x][0]);
                        o2[x][1] = fma2(S[2 * j + 1][x], qq.y, o2[x][1]);
                    }
                }
                const float beta = sb[tt], kq = sb[s.chunk + tt];
                float u[CPT], o[CPT];
#pragma unroll
                for (int x = 0; x < CPT; ++x) {
                    const float2 ms = unpack2(add2(m2[x][0], m2[x][1])), os = unpack2(add2(o2[x][0], o2[x][1]));
                    float m = ms.x + ms.y;
                    o[x] = os.x + os.y;
                    m += __shfl_xor_sync(0xffffffffu, m, 8);
                    o[x] += __shfl_xor_sync(0xffffffffu, o[x], 8);
                    m += __shfl_xor_sync(0xffffffffu, m, 16);
                    o[x] += __shfl_xor_sync(0xffffffffu, o[x], 16);
                    u[x] = beta * (sv[tt * s.cols + x] - m);
                    o[x] = fmaf(kq, u[x], o[x]);
                }
#pragma unroll
                for (int x = 0; x < CPT; ++x) {
                    const f32x2 uu = pack2(u[x], u[x]);
#pragma unroll
                    for (int i = 0; i < RL / 2; ++i) S[i][x] = fma2(k2[i], uu, S[i][x]);
                }
                if (rg == 0) {
                    if constexpr (CPT == 2) *reinterpret_cast<float2*>(ys + tt * s.cols) = make_float2(o[0], o[1]);
                    else ys[tt * s.cols] = o[0];
                }
            }
        } else {
            const int w = warp - s.consumers, nw = nwarps - s.consumers;
            if (c + 1 < chunks) stage(c + 1, w, nw);
            if (c > 0) finish(c - 1, w, nw);
        }
        barrier();
    }
    if (consumer) {
        if (mine) {
#pragma unroll
            for (int i = 0; i < RL / 2; ++i) {
                const int r = (i >> 1) * 16 + rg * 4 + (i & 1) * 2;
                if (r < p.dk) {
                    if constexpr (CPT == 2) {
                        const float2 a = unpack2(S[i][0]), d = unpack2(S[i][1]);
                        *reinterpret_cast<float2*>(state + (size_t)r * p.dv) = make_float2(a.x, d.x);
                        *reinterpret_cast<float2*>(state + (size_t)(r + 1) * p.dv) = make_float2(a.y, d.y);
                    } else {
                        const float2 a = unpack2(S[i][0]);
                        state[(size_t)r * p.dv] = a.x;
                        state[(size_t)(r + 1) * p.dv] = a.y;
                    }
                }
            }
        }
    } else {
        finish(chunks - 1, warp - s.consumers, nwarps - s.consumers);
    }
    if (s.parts > 1) cluster.sync();       // the other parts may still read this CTA's read-outs
}

template <class E, int RL, int CPT>
int launch_channel_delta(const ovb_delta_args& a, cudaStream_t stream) {
    DeltaShape s;
    const int unit = 8 * CPT, groups = ceil_div(a.dv, unit);       // column groups of a warp each
    // one CTA per (sequence, head) when those fill the machine, else up to eight that share the columns
    s.parts = 1;
    while (s.parts < 8 && a.B * a.H * s.parts * 2 <= 148 && ceil_div(groups, s.parts * 2) * unit * (s.parts * 2 - 1) < a.dv) s.parts *= 2;
    while (ceil_div(groups, s.parts) > 8) s.parts *= 2;
    s.consumers = ceil_div(groups, s.parts);
    s.cols = s.consumers * unit;
    if (s.parts > 8) {
        set_error("ovb_channel_delta: value size %d is too large", a.dv);
        return ERR_UNSUPPORTED;
    }
    s.chunk = a.max_q_len == 1 ? 1 : RL <= 32 ? 16 : 8;
    const int producers = a.max_q_len == 1 ? 2 : s.consumers <= 4 ? 8 : 4;      // at most 12 warps
    const int dp = RL * 4;
    const size_t smem = 4 * ((size_t)2 * stage_floats(dp, s.cols, s.chunk) + 2 * s.chunk * s.cols + a.taps * (2 * dp + s.cols) + dp + s.cols);
    OVB_REQUIRE(smem <= 227 * 1024, "ovb_channel_delta: %d taps need too much shared memory", a.taps);
    auto kern = channel_delta_kernel<E, RL, CPT>;
    static std::atomic<uint64_t> configured{0};
    int dev = 0;
    OVB_CHECK_CUDA(cudaGetDevice(&dev));
    const uint64_t bit = 1ull << (dev & 63);
    if (!(configured.load(std::memory_order_acquire) & bit)) {
        OVB_CHECK_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
        configured.fetch_or(bit, std::memory_order_release);
    }
    cudaLaunchConfig_t cfg;
    memset(&cfg, 0, sizeof(cfg));
    cfg.gridDim = dim3(a.H * s.parts, a.B);
    cfg.blockDim = dim3((s.consumers + producers) * 32);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[2];
    int n = 0;
    if (s.parts > 1) {
        attr[n].id = cudaLaunchAttributeClusterDimension;
        attr[n].val.clusterDim.x = s.parts;
        attr[n].val.clusterDim.y = attr[n].val.clusterDim.z = 1;
        ++n;
    }
    if (pdl_enabled()) {
        attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[n].val.programmaticStreamSerializationAllowed = 1;
        ++n;
    }
    cfg.attrs = attr;
    cfg.numAttrs = n;
    OVB_CHECK_CUDA(cudaLaunchKernelEx(&cfg, kern, a, s));
    return 0;
}

}  // namespace

}  // namespace ovb

extern "C" int ovb_channel_delta(const ovb_delta_args* a, ovb_stream_t stream_) {
    using namespace ovb;
    cudaStream_t stream = (cudaStream_t)stream_;
    OVB_REQUIRE(a && a->proj && a->low && a->conv_w && a->conv_ring && a->decay_a && a->dt_bias && a->norm && a->state && a->out && a->subsequence_begins &&
                    a->past_lens && a->slots, "ovb_channel_delta: null operand");
    OVB_REQUIRE(a->B > 0 && a->B <= 65535 && a->T > 0 && a->G > 0 && a->H > 0 && a->H % a->G == 0 && a->taps > 0 && a->D > 0 && a->Dv > 0 && a->dk >= a->D &&
                    a->dv >= a->Dv, "ovb_channel_delta: bad sizes");
    auto aligned = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
    OVB_REQUIRE(a->dk % 16 == 0 && a->dv % 16 == 0 && a->ldp % 4 == 0 && a->k_off % 4 == 0 && a->v_off % 4 == 0 && a->ld_low % 4 == 0 && a->gate_off % 4 == 0 &&
                    a->conv_cols % 4 == 0 && a->conv_cols >= a->v_off + a->H * a->dv && a->ldo % 4 == 0 && a->o_head % 4 == 0,
                "ovb_channel_delta: heads must be padded to 16 columns, pitches to 4");
    OVB_REQUIRE(aligned(a->proj) && aligned(a->low) && aligned(a->conv_w) && aligned(a->conv_ring) && aligned(a->dt_bias) && aligned(a->state) && aligned(a->out),
                "ovb_channel_delta: operands must be 16-byte aligned");
    return dispatch_store(a->dtype, "ovb_channel_delta", [&](auto e) -> int {
        using E = decltype(e);
        if (a->dk <= 32) return launch_channel_delta<E, 8, 2>(*a, stream);
        if (a->dk <= 64) return launch_channel_delta<E, 16, 2>(*a, stream);
        if (a->dk <= 128) return launch_channel_delta<E, 32, 2>(*a, stream);
        if (a->dk <= 256) return launch_channel_delta<E, 64, 1>(*a, stream);
        set_error("ovb_channel_delta: key size %d above 256", a->dk);
        return ERR_UNSUPPORTED;
    });
}
