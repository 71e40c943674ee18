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
// One CTA works on (sequence, head, part of the columns). Consumer warps run the recurrence over a stage of up to 16 tokens in shared
// memory; producer warps meanwhile fetch the raw inputs two stages ahead (cp.async), prepare the next stage (convolution, silu, norms,
// decays: one warp per token) and finish the previous one (norm of the read-out, gate, store). When there are too few (sequence, head) pairs to fill the machine, a cluster of CTAs shares a
// head's columns and reads each other's read-outs through distributed shared memory for the norm. Decode steps have a kernel of their own.
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

template <class E>
__device__ __forceinline__ float4 silu4(float4 z) {
    return make_float4(z.x * Fn<E>::sigmoid(z.x), z.y * Fn<E>::sigmoid(z.y), z.z * Fn<E>::sigmoid(z.z), z.w * Fn<E>::sigmoid(z.w));
}
template <class E>
__device__ __forceinline__ float4 sigmoid4(float4 z) {
    return make_float4(Fn<E>::sigmoid(z.x), Fn<E>::sigmoid(z.y), Fn<E>::sigmoid(z.z), Fn<E>::sigmoid(z.w));
}
__device__ __forceinline__ float dot4(float4 a, float4 b) { return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, a.w * b.w))); }
__device__ __forceinline__ float4 mul4(float4 a, float4 b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }
__device__ __forceinline__ float4 scale4(float4 a, float c) { return make_float4(a.x * c, a.y * c, a.z * c, a.w * c); }
template <class E>
__device__ __forceinline__ float4 decay4(float a, float4 low, float4 bias) {
    return make_float4(expf(-a * Fn<E>::softplus(low.x + bias.x)), expf(-a * Fn<E>::softplus(low.y + bias.y)), expf(-a * Fn<E>::softplus(low.z + bias.z)),
                       expf(-a * Fn<E>::softplus(low.w + bias.w)));
}

struct DeltaShape {
    int parts;               // CTAs that share a head's columns (a cluster)
    int cols;                // columns per CTA, a multiple of 8 CPT (the last part may reach past dv)
    int consumers;           // warps that run the recurrence: cols / (8 CPT)
    int chunk;               // tokens per stage
};

// Floats of one stage: K, Q, G [chunk][DP], V [chunk][cols], beta and k . q [chunk] (padded to whole 16-byte pieces).
__host__ __device__ inline int stage_floats(int dp, int cols, int chunk) { return chunk * (3 * dp + cols) + (2 * chunk + 3) / 4 * 4; }
// Bytes of the raw inputs of one stage: rows of the head's q, k and of this CTA's v columns (chunk + taps - 1 tokens), decay inputs (chunk tokens).
__host__ __device__ inline int raw_bytes(int dk, int cols, int chunk, int taps, int elem) { return (chunk + taps - 1) * (2 * dk + cols) * elem + chunk * dk * 4; }

__device__ __forceinline__ void copy16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void copy_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void copy_wait() {
    asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

// Warps of a CTA: fewer where the state takes more registers.
constexpr int max_warps(int rl) { return rl >= 64 ? 10 : 12; }

template <class E, int RL, int CPT>
__global__ void __launch_bounds__(max_warps(RL) * 32, 1) channel_delta_kernel(ovb_delta_args p, DeltaShape s) {
    constexpr int DP = RL * 4;                     // rows, zero behind p.dk
    constexpr int NV = (DP + 127) / 128;           // pieces of four rows per lane
    extern __shared__ __align__(16) float smem[];
    const int stage_len = stage_floats(DP, s.cols, s.chunk);
    float* y_buf = smem + 2 * stage_len;           // [2][chunk][cols] read-outs
    float* s_conv = y_buf + 2 * s.chunk * s.cols;  // [taps][2 DP + cols] filters of the head's q, k and of this CTA's v columns
    const int conv_len = 2 * DP + s.cols;
    float* s_bias = s_conv + p.taps * conv_len;    // [DP]
    float* s_norm = s_bias + DP;                   // [cols]
    uint8_t* raw_buf = reinterpret_cast<uint8_t*>(s_norm + s.cols);      // [2] raw inputs
    const int raw_len = raw_bytes(p.dk, s.cols, s.chunk, p.taps, sizeof(E)), raw_pitch = 2 * p.dk + s.cols, keep = p.taps - 1;

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int part = blockIdx.x % s.parts, h = blockIdx.x / s.parts, b = blockIdx.y;
    const int c0 = part * s.cols, kvh = h / (p.H / p.G);
    const bool consumer = warp < s.consumers;
    const int pw = warp - s.consumers, npw = (blockDim.x >> 5) - s.consumers;       // producer warps
    const int pt = threadIdx.x - s.consumers * 32, npt = npw * 32;
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
    const int chunks = (len + s.chunk - 1) / s.chunk;
    const E* proj = reinterpret_cast<const E*>(p.proj);
    const int q_col = kvh * p.dk, k_col = p.k_off + kvh * p.dk, v_col = p.v_off + h * p.dv + c0;
    const int v_cols = max(0, min(s.cols, p.dv - c0));
    __syncthreads();

    // raw inputs of stage c, on their way: row r of the buffer is token c * chunk - keep + r of the piece
    auto fetch = [&](int c) {
        constexpr int EPC = 16 / sizeof(E);        // elements per 16-byte piece
        E* rows = reinterpret_cast<E*>(raw_buf + (c & 1) * raw_len);
        float* low = reinterpret_cast<float*>(rows + (s.chunk + keep) * raw_pitch);
        const int first = c * s.chunk - keep, n = min(s.chunk, len - c * s.chunk);
        const int nk = p.dk / EPC, per_row = 2 * nk + v_cols / EPC;
        for (int i = pt; i < (n + keep) * per_row; i += npt) {
            const int r = i / per_row, x = i % per_row, rel = first + r;
            const int dst = x < 2 * nk ? x * EPC : 2 * p.dk + (x - 2 * nk) * EPC;
            const int col = x < nk ? q_col + x * EPC : x < 2 * nk ? k_col + (x - nk) * EPC : v_col + (x - 2 * nk) * EPC;
            E* d = rows + r * raw_pitch + dst;
            if (rel >= 0) {
                copy16(d, proj + (size_t)(begin + rel) * p.ldp + col);
            } else {                               // before this piece: what earlier steps left, or zeros before position 0
                const int pos = past + rel;
                const float* ring = p.conv_ring + ((size_t)slot * p.taps + (pos >= 0 ? pos % p.taps : 0)) * p.conv_cols + col;
#pragma unroll
                for (int e = 0; e < EPC; ++e) st_f32(d + e, pos >= 0 ? ring[e] : 0.f);
            }
        }
        const int nl = p.dk / 4;
        for (int i = pt; i < n * nl; i += npt)
            copy16(low + (i / nl) * p.dk + (i % nl) * 4, p.low + (size_t)(begin + c * s.chunk + i / nl) * p.ld_low + (size_t)h * p.dk + (i % nl) * 4);
    };
    // stage c from its raw inputs, a warp per token
    auto stage = [&](int c) {
        const E* rows = reinterpret_cast<const E*>(raw_buf + (c & 1) * raw_len);
        const float* low = reinterpret_cast<const float*>(rows + (s.chunk + keep) * raw_pitch);
        float* st = smem + (c & 1) * stage_len;
        const int n = min(s.chunk, len - c * s.chunk);
        for (int tt = pw; tt < n; tt += npw) {
            const float bl = lane == 0 ? ld_f32(proj + (size_t)(begin + c * s.chunk + tt) * p.ldp + p.b_off + h) : 0.f;
            const E* in = rows + tt * raw_pitch;
            float4 q[NV], k[NV];
            float qq = 0.f, kk = 0.f, qk = 0.f;
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const int x = i * 128 + lane * 4;
                q[i] = k[i] = make_float4(0.f, 0.f, 0.f, 0.f);
                if (x < p.dk) {
#pragma unroll 2
                    for (int j = 0; j < p.taps; ++j) {
                        q[i] = fma4(ld4_f32(s_conv + j * conv_len + x), ld4_f32(in + j * raw_pitch + x), q[i]);
                        k[i] = fma4(ld4_f32(s_conv + j * conv_len + DP + x), ld4_f32(in + j * raw_pitch + p.dk + x), k[i]);
                    }
                    q[i] = silu4<E>(q[i]);
                    k[i] = silu4<E>(k[i]);
                }
                qq += dot4(q[i], q[i]);
                kk += dot4(k[i], k[i]);
                qk += dot4(q[i], k[i]);
            }
            const float iq = p.q_scale / sqrtf(delta_sum(qq) + 1e-6f), ik = 1.f / sqrtf(delta_sum(kk) + 1e-6f);
            qk = delta_sum(qk) * iq * ik;
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const int x = i * 128 + lane * 4;
                if (x < DP) {
                    const float4 g = x < p.dk ? decay4<E>(decay_a, ld4_f32(low + tt * p.dk + x), ld4_f32(s_bias + x)) : make_float4(1.f, 1.f, 1.f, 1.f);
                    st4_f32(st + tt * DP + x, scale4(k[i], ik));
                    st4_f32(st + (s.chunk + tt) * DP + x, scale4(q[i], iq));
                    st4_f32(st + (2 * s.chunk + tt) * DP + x, g);
                }
            }
            for (int x = lane * 4; x < s.cols; x += 128) {
                float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
                if (x < v_cols) {
#pragma unroll 4
                    for (int j = 0; j < p.taps; ++j)
                        v = fma4(ld4_f32(s_conv + j * conv_len + 2 * DP + x), ld4_f32(in + j * raw_pitch + 2 * p.dk + x), v);
                    v = silu4<E>(v);
                }
                st4_f32(st + 3 * s.chunk * DP + tt * s.cols + x, v);
            }
            if (lane == 0) {
                st[s.chunk * (3 * DP + s.cols) + tt] = Fn<E>::sigmoid(bl);
                st[s.chunk * (3 * DP + s.cols) + s.chunk + tt] = qk;
            }
        }
    };
    // norm, gate and store of the read-outs of stage c; columns of the other parts of the cluster are read for the norm only
    auto finish = [&](int c) {
        const int n = min(s.chunk, len - c * s.chunk);
        const float* ys = y_buf + (c & 1) * s.chunk * s.cols;
        const float* gate = p.low + (size_t)(begin + c * s.chunk) * p.ld_low + p.gate_off + (size_t)h * p.dv + c0;
        E* out = reinterpret_cast<E*>(p.out) + (size_t)(begin + c * s.chunk) * p.ldo + (size_t)h * p.o_head + c0;
        const int x = lane * 4;
        float4 g = pw < n && x < v_cols ? ld4_f32(gate + (size_t)pw * p.ld_low + x) : make_float4(0.f, 0.f, 0.f, 0.f);
        for (int tt = pw; tt < n; tt += npw) {
            const float4 g_now = g;
            if (tt + npw < n && x < v_cols) g = ld4_f32(gate + (size_t)(tt + npw) * p.ld_low + x);        // (the next token's, ahead of its use)
            float ss = 0.f;
            for (int col = x; col < s.parts * s.cols; col += 128) {
                const int from = col / s.cols;
                const float* row = ys + tt * s.cols + (col - from * s.cols);
                const float4 y = ld4_f32(from == part ? row : cluster.map_shared_rank(row, from));
                ss += dot4(y, y);
            }
            const float inv = 1.f / sqrtf(delta_sum(ss) / (float)p.Dv + p.eps);
            for (int col = x; col < v_cols; col += 128) {
                const float4 gv = col == x ? g_now : ld4_f32(gate + (size_t)tt * p.ld_low + col);
                st4_f32(out + (size_t)tt * p.ldo + col, mul4(scale4(mul4(ld4_f32(ys + tt * s.cols + col), ld4_f32(s_norm + col)), inv), sigmoid4<E>(gv)));
            }
        }
    };
    auto producers_meet = [&]() { asm volatile("bar.sync 1, %0;" ::"r"(npt) : "memory"); };

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
        fetch(0);
        copy_commit();
        if (chunks > 1) fetch(1);
        copy_commit();
        copy_wait<1>();
        producers_meet();
        stage(0);
    }
    barrier();
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
            if (c + 2 < chunks) fetch(c + 2);      // (into the buffer of stage c, which is finished)
            copy_commit();
            if (c + 1 < chunks) {
                copy_wait<1>();
                producers_meet();
                stage(c + 1);
            }
            if (c > 0) finish(c - 1);
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
        finish(chunks - 1);
    }
    if (s.parts > 1) cluster.sync();       // the other parts may still read this CTA's read-outs
}

// One token per sequence (decoding): a CTA per (sequence, head) whose threads hold four columns at up to RT rows each. The state is
// requested first and arrives while a few warps prepare the token; sums over the row groups pass through shared memory.
constexpr int STEP_THREADS = 256, STEP_FINISH = 4;      // STEP_FINISH: the warp that norms and gates the read-out

template <class E, int RT>
__global__ void __launch_bounds__(STEP_THREADS, RT <= 4 ? 3 : 2) channel_delta_step_kernel(ovb_delta_args p) {
    extern __shared__ __align__(16) float smem[];
    const int cgs = p.dv / 4, rgs = STEP_THREADS / cgs;            // column groups, row groups
    float* s_k = smem;                          // [dk] each
    float* s_q = s_k + p.dk;
    float* s_g = s_q + p.dk;
    float* s_v = s_g + p.dk;                    // [dv]
    float* s_m = s_v + p.dv;                    // [rgs][dv] partial sums of S^T k, then of S^T q
    float* s_o = s_m + rgs * p.dv;
    float* s_one = s_o + rgs * p.dv;            // beta, k . q
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h = blockIdx.x, b = blockIdx.y, kvh = h / (p.H / p.G), keep = p.taps - 1;
    const int cg4 = threadIdx.x % cgs * 4, rg = threadIdx.x / cgs;
    const bool live = rg < rgs;
    pdl_enter();
    const int t = p.subsequence_begins[b], past = p.past_lens[b], slot = p.slots[b];
    float* state = p.state + ((size_t)slot * p.H + h) * p.dk * p.dv + cg4;
    float4 S[RT];                                // rows rg, rg + rgs, ...
#pragma unroll
    for (int i = 0; i < RT; ++i) {
        const int r = rg + i * rgs;
        S[i] = live && r < p.dk && past > 0 ? ld4_f32(state + (size_t)r * p.dv) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const E* row = reinterpret_cast<const E*>(p.proj) + (size_t)t * p.ldp;
    float* ring = p.conv_ring + (size_t)slot * p.taps * p.conv_cols;
    auto conv = [&](int col, bool store) {
        const float4 now = ld4_f32(row + col);
        float4 acc = mul4(ld4_f32(p.conv_w + (size_t)keep * p.conv_cols + col), now);
#pragma unroll 3
        for (int j = 0; j < keep; ++j) {
            const int pos = past - keep + j;
            if (pos >= 0) acc = fma4(ld4_f32(p.conv_w + (size_t)j * p.conv_cols + col), ld4_f32(ring + (size_t)(pos % p.taps) * p.conv_cols + col), acc);
        }
        if (store && keep > 0) st4_f32(ring + (size_t)(past % p.taps) * p.conv_cols + col, now);
        return silu4<E>(acc);
    };
    constexpr int NV = 2;                        // dk, dv up to 256
    float4 gate[NV];
    if (warp == 0) {
        float4 q[NV], k[NV];
        float qq = 0.f, kk = 0.f, qk = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int x = i * 128 + lane * 4;
            q[i] = k[i] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (x < p.dk) {
                const bool owner = h % (p.H / p.G) == 0;
                q[i] = conv(kvh * p.dk + x, owner);
                k[i] = conv(p.k_off + kvh * p.dk + x, owner);
            }
            qq += dot4(q[i], q[i]);
            kk += dot4(k[i], k[i]);
            qk += dot4(q[i], k[i]);
        }
        const float iq = p.q_scale / sqrtf(delta_sum(qq) + 1e-6f), ik = 1.f / sqrtf(delta_sum(kk) + 1e-6f);
        qk = delta_sum(qk) * iq * ik;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int x = i * 128 + lane * 4;
            if (x < p.dk) {
                st4_f32(s_q + x, scale4(q[i], iq));
                st4_f32(s_k + x, scale4(k[i], ik));
            }
        }
        if (lane == 0) s_one[1] = qk;
    } else if (warp == 1) {
        const float a = p.decay_a[h];
        for (int x = lane * 4; x < p.dk; x += 128)
            st4_f32(s_g + x, decay4<E>(a, ld4_f32(p.low + (size_t)t * p.ld_low + (size_t)h * p.dk + x), ld4_f32(p.dt_bias + (size_t)h * p.dk + x)));
    } else if (warp == 2) {
        for (int x = lane * 4; x < p.dv; x += 128) st4_f32(s_v + x, conv(p.v_off + h * p.dv + x, true));
    } else if (warp == STEP_FINISH) {
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int x = i * 128 + lane * 4;
            gate[i] = x < p.dv ? ld4_f32(p.low + (size_t)t * p.ld_low + p.gate_off + (size_t)h * p.dv + x) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    } else if (warp == 3 && lane == 0) {
        s_one[0] = Fn<E>::sigmoid(ld_f32(row + p.b_off + h));
    }
    __syncthreads();
    if (live) {
        float4 m = make_float4(0.f, 0.f, 0.f, 0.f), o = m;
#pragma unroll
        for (int i = 0; i < RT; ++i) {
            const int r = rg + i * rgs;
            if (r < p.dk) {
                const float g = s_g[r], k = s_k[r], q = s_q[r];
                S[i] = scale4(S[i], g);
                m = fma4(S[i], make_float4(k, k, k, k), m);
                o = fma4(S[i], make_float4(q, q, q, q), o);
            }
        }
        st4_f32(s_m + rg * p.dv + cg4, m);
        st4_f32(s_o + rg * p.dv + cg4, o);
    }
    __syncthreads();
    const float beta = s_one[0], kq = s_one[1];
    auto step_of = [&](int col) {                // u of four columns
        float4 m = ld4_f32(s_m + col);
        for (int r = 1; r < rgs; ++r) {
            const float4 x = ld4_f32(s_m + r * p.dv + col);
            m = make_float4(m.x + x.x, m.y + x.y, m.z + x.z, m.w + x.w);
        }
        const float4 v = ld4_f32(s_v + col);
        return make_float4(beta * (v.x - m.x), beta * (v.y - m.y), beta * (v.z - m.z), beta * (v.w - m.w));
    };
    if (live) {
        const float4 u = step_of(cg4);
#pragma unroll
        for (int i = 0; i < RT; ++i) {
            const int r = rg + i * rgs;
            if (r < p.dk) {
                const float k = s_k[r];
                st4_f32(state + (size_t)r * p.dv, fma4(make_float4(k, k, k, k), u, S[i]));
            }
        }
    }
    if (warp == STEP_FINISH) {
        float4 y[NV];
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int x = i * 128 + lane * 4;
            y[i] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (x < p.dv) {
                y[i] = scale4(step_of(x), kq);
                for (int r = 0; r < rgs; ++r) {
                    const float4 o = ld4_f32(s_o + r * p.dv + x);
                    y[i] = make_float4(y[i].x + o.x, y[i].y + o.y, y[i].z + o.z, y[i].w + o.w);
                }
            }
            ss += dot4(y[i], y[i]);
        }
        const float inv = 1.f / sqrtf(delta_sum(ss) / (float)p.Dv + p.eps);
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int x = i * 128 + lane * 4;
            if (x < p.dv)
                st4_f32(reinterpret_cast<E*>(p.out) + (size_t)t * p.ldo + (size_t)h * p.o_head + x,
                        mul4(scale4(mul4(y[i], ld4_f32(p.norm + x)), inv), sigmoid4<E>(gate[i])));
        }
    }
}

// Decode steps of the sizes that the kernel above holds in registers; ERR_UNSUPPORTED otherwise.
template <class E>
int launch_channel_delta_step(const ovb_delta_args& a, cudaStream_t stream) {
    if (a.max_q_len != 1 || a.T != a.B || a.dk > 256 || a.dv > 256) return ERR_UNSUPPORTED;
    const int rgs = STEP_THREADS / (a.dv / 4), rows = ceil_div(a.dk, rgs);
    const size_t smem = 4 * (size_t)(3 * a.dk + a.dv + 2 * rgs * a.dv + 4);
    auto go = [&](auto kern) -> int {
        OVB_CHECK_CUDA(launch_pdl(kern, dim3(a.H, a.B), dim3(STEP_THREADS), smem, stream, a));
        return 0;
    };
    if (rows <= 4) return go(channel_delta_step_kernel<E, 4>);
    if (rows <= 8) return go(channel_delta_step_kernel<E, 8>);
    if (rows <= 16) return go(channel_delta_step_kernel<E, 16>);
    return ERR_UNSUPPORTED;
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
    const int dp = RL * 4;
    auto bytes = [&]() {
        return 4 * ((size_t)2 * stage_floats(dp, s.cols, s.chunk) + 2 * s.chunk * s.cols + a.taps * (2 * dp + s.cols) + dp + s.cols) +
               2 * (size_t)raw_bytes(a.dk, s.cols, s.chunk, a.taps, sizeof(E));
    };
    s.chunk = a.max_q_len == 1 ? 1 : 16;
    while (s.chunk > 1 && bytes() > 227 * 1024) s.chunk /= 2;
    const size_t smem = bytes();
    OVB_REQUIRE(smem <= 227 * 1024, "ovb_channel_delta: %d taps need too much shared memory", a.taps);
    const int producers = a.max_q_len == 1 ? 2 : max_warps(RL) - s.consumers < 8 ? max_warps(RL) - s.consumers : 8;
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
    return update_conv_ring<E>(a.proj, a.ldp, {a.conv_w, a.conv_ring, a.taps, a.conv_cols}, a.subsequence_begins, a.past_lens, a.slots, a.B, stream);
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
        const int rc = launch_channel_delta_step<E>(*a, stream);
        if (rc != ERR_UNSUPPORTED) return rc;
        if (a->dk <= 32) return launch_channel_delta<E, 8, 2>(*a, stream);
        if (a->dk <= 64) return launch_channel_delta<E, 16, 2>(*a, stream);
        if (a->dk <= 128) return launch_channel_delta<E, 32, 2>(*a, stream);
        if (a->dk <= 256) return launch_channel_delta<E, 64, 1>(*a, stream);
        set_error("ovb_channel_delta: key size %d above 256", a->dk);
        return ERR_UNSUPPORTED;
    });
}
