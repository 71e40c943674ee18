// Gated delta rule with a decay per key channel, fused with everything between its projections and the output projection: short
// convolutions, silu, unit norms, decays, step sizes, the recurrence, the norm of its read-out and the output gate.
//
// The state S [dk, dv] of a head lives in registers and touches memory twice per step. A token reads it, then changes it:
//
//     S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//
// Prompts take four tokens at a time. With c_t = g_1 .. g_t (products of decays, never quotients: nothing overflows),
//
//     u_t = beta_t (v_t - S^T (c_t k_t) - sum_{s<t} A_ts u_s),      A_ts = k_t . (g_{s+1} .. g_t k_s)
//     o_t = S^T (c_t q_t) + sum_{s<=t} B_ts u_s,                    B_ts = q_t . (g_{s+1} .. g_t k_s)
//     S   <- c_4 S + sum_s (g_{s+1} .. g_4 k_s) u_s^T
//
// and with w_t = v_t - S^T (c_t k_t) the first two lines are u = U w, o = S^T c q + O w for two small triangular matrices,
// U = (I + diag(beta) A)^-1 diag(beta) and O = B U; which is the same sum in another order, entirely in fp32: 13 operations per state
// element for four tokens instead of 16, and one reduction over the rows instead of four behind one another. Everything that does not
// depend on the state (convolutions, silu, unit norms, decays, the vectors and matrices above) is prepared by a kernel that works on all
// groups of four at once (delta_prepare_kernel); the recurrence itself (delta_scan_kernel) walks the groups of a sequence.
//
// Columns of the state are independent: a consumer warp of the scan owns some of them, and no barrier of the CTA stands in a group's
// chain. With bf16 storage the products run on the tensor cores with every fp32 operand split into two tf32 parts (MmaState), with fp32
// storage on the fp32 units (FmaState). Producer warps fetch the next stage of groups (bulk copies) and finish the previous one (norm of
// the read-out, gate, store). When there are too few (sequence, head) pairs to fill the machine, a cluster of CTAs shares a head's columns
// and reads each other's read-outs through distributed shared memory for the norm, and teams of warps share the rows. Decode steps have a
// kernel of their own.
#include <cooperative_groups.h>

#include <atomic>

#include "common.cuh"
#include "short_conv.cuh"
#include "sm100_ptx.cuh"
#include "store_types.cuh"
#include "warp_sums.cuh"

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

constexpr int GROUP = 4;                // tokens taken at a time
constexpr int GROUP_SCALARS = 2 * GROUP * GROUP;                  // U and O, lower triangles row by row
static_assert(GROUP == 4, "a row of U or O is one 16-byte piece");

// The record of one (group, head) as the scan reads it: vectors c_t k_t and c_t q_t of dp rows (zeros from dk on) at a pitch of kq floats,
// decayed k_s at a pitch of kd, c_4, U and O, values [4][dv]. A sequence whose tokens of this step begin at row t has its groups in rows
// t / 4 + b, ... (they do not overlap: T / 4 + B rows are enough).
struct RecordLayout {
    int dp, kq, kd;
    __host__ __device__ int decayed() const { return 2 * GROUP * kq; }
    __host__ __device__ int all() const { return decayed() + GROUP * kd; }
    __host__ __device__ int scalars() const { return all() + dp; }
    __host__ __device__ int values() const { return scalars() + GROUP_SCALARS; }
    __host__ __device__ int floats(int dv) const { return values() + GROUP * dv; }
};
__device__ __forceinline__ int first_group(const int* begins, int b) { return begins[b] / GROUP + b; }

// One warp per (group, head). TAPS 0: any number of taps.
template <class E, int NV, int TAPS>
__global__ void __launch_bounds__(128) delta_prepare_kernel(ovb_delta_args p, RecordLayout lay) {
    pdl_enter();
    __shared__ int s_b;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row = blockIdx.x, h = blockIdx.y * 4 + warp;
    for (int b = threadIdx.x; b < p.B; b += 128)
        if (first_group(p.subsequence_begins, b) <= row && row < first_group(p.subsequence_begins, b + 1)) s_b = b;
    __syncthreads();
    const int b = s_b, begin = p.subsequence_begins[b], len = p.subsequence_begins[b + 1] - begin;
    const int t0 = (row - first_group(p.subsequence_begins, b)) * GROUP, n = min(GROUP, len - t0);      // tokens of the group
    if (n <= 0 || h >= p.H) return;
    const int past = p.past_lens[b], kvh = h / (p.H / p.G);
    const E* proj = reinterpret_cast<const E*>(p.proj);
    const ShortConv cv = {p.conv_w, p.conv_ring, TAPS > 0 ? TAPS : p.taps, p.conv_cols};
    const float* ring = p.conv_ring + (size_t)p.slots[b] * cv.taps * cv.cols;
    float* rec = p.records + ((size_t)row * p.H + h) * lay.floats(p.dv);
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);

    // convolution and silu of four columns for the tokens of the group; zeros behind the last token
    auto conv = [&](int col, float4 (&y)[GROUP]) {
        if constexpr (TAPS > 0) {
            Raw4<E> in[TAPS + GROUP - 1];
            float4 w[TAPS];
#pragma unroll
            for (int j = 0; j < TAPS + GROUP - 1; ++j) {
                const int rel = t0 + j - (TAPS - 1);
                if (rel >= 0 && rel < len) in[j].load(proj + (size_t)(begin + rel) * p.ldp + col);
                else if (rel < 0 && past + rel >= 0) in[j].set(ld4_f32(ring + (size_t)((past + rel) % TAPS) * cv.cols + col));
                else in[j].set(zero);
            }
#pragma unroll
            for (int j = 0; j < TAPS; ++j) w[j] = ld4_f32(p.conv_w + (size_t)j * cv.cols + col);
#pragma unroll
            for (int t = 0; t < GROUP; ++t) {
                float4 acc = zero;
#pragma unroll
                for (int j = 0; j < TAPS; ++j) acc = fma4(w[j], in[t + j].get(), acc);
                y[t] = t < n ? silu4<E>(acc) : zero;
            }
        } else {
#pragma unroll
            for (int t = 0; t < GROUP; ++t) {
                float4 acc = zero;
                if (t < n)
                    for (int j = 0; j < cv.taps; ++j)
                        acc = fma4(ld4_f32(cv.w + (size_t)j * cv.cols + col),
                                   conv_input4(proj + col, p.ldp, ring + col, cv, begin + t0 + t, begin, past + t0 + t, cv.taps - 1 - j), acc);
                y[t] = silu4<E>(acc);
            }
        }
    };
    float4 q[NV][GROUP], k[NV][GROUP];
    float sums[2 * GROUP] = {};
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = i * 128 + lane * 4;
        if (c < p.dk) {
            conv(kvh * p.dk + c, q[i]);
            conv(p.k_off + kvh * p.dk + c, k[i]);
        } else {
#pragma unroll
            for (int t = 0; t < GROUP; ++t) q[i][t] = k[i][t] = zero;
        }
#pragma unroll
        for (int t = 0; t < GROUP; ++t) {
            sums[t] += dot4(q[i][t], q[i][t]);
            sums[GROUP + t] += dot4(k[i][t], k[i][t]);
        }
    }
    const float total = rec_reduce8(sums, lane);
    float scale[2 * GROUP];
#pragma unroll
    for (int j = 0; j < 2 * GROUP; ++j)
        scale[j] = (j < GROUP ? p.q_scale : 1.f) / sqrtf(__shfl_sync(0xffffffffu, total, ((j & 1) << 4) | ((j >> 1 & 1) << 3) | ((j >> 2 & 1) << 2)) + 1e-6f);
    float ab[16] = {};                            // A then B
    const float a = p.decay_a[h];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = i * 128 + lane * 4;
        if (c >= p.dk) {
            if (c < lay.dp) {
#pragma unroll
                for (int t = 0; t < 2 * GROUP; ++t) st4_f32(rec + t * lay.kq + c, zero);
#pragma unroll
                for (int t = 0; t < GROUP; ++t) st4_f32(rec + lay.decayed() + t * lay.kd + c, zero);
                st4_f32(rec + lay.all() + c, zero);
            }
            continue;
        }
        const float4 bias = ld4_f32(p.dt_bias + (size_t)h * p.dk + c);
        float4 g[GROUP], r[GROUP], all = make_float4(1.f, 1.f, 1.f, 1.f);
#pragma unroll
        for (int t = 0; t < GROUP; ++t)
            g[t] = t < n ? decay4<E>(a, ld4_f32(p.low + (size_t)(begin + t0 + t) * p.ld_low + (size_t)h * p.dk + c), bias) : make_float4(1.f, 1.f, 1.f, 1.f);
#pragma unroll
        for (int t = 0; t < GROUP; ++t) {
            const float4 kt = scale4(k[i][t], scale[GROUP + t]), qt = scale4(q[i][t], scale[t]);
            all = mul4(all, g[t]);
            st4_f32(rec + t * lay.kq + c, mul4(all, kt));
            st4_f32(rec + (GROUP + t) * lay.kq + c, mul4(all, qt));
#pragma unroll
            for (int s = 0; s < t; ++s) {
                r[s] = mul4(r[s], g[t]);
                ab[t * (t - 1) / 2 + s] += dot4(kt, r[s]);
                ab[6 + t * (t + 1) / 2 + s] += dot4(qt, r[s]);
            }
            r[t] = kt;
            ab[6 + t * (t + 1) / 2 + t] += dot4(qt, kt);
        }
#pragma unroll
        for (int s = 0; s < GROUP; ++s) st4_f32(rec + lay.decayed() + s * lay.kd + c, r[s]);
        st4_f32(rec + lay.all() + c, all);
    }
    // U and O, by every lane; beta of tokens behind the last is zero
    const float beta = lane < n ? Fn<E>::sigmoid(ld_f32(proj + (size_t)(begin + t0 + lane) * p.ldp + p.b_off + h)) : 0.f;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        float v[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = ab[half * 8 + j];
        const float sum = rec_reduce8(v, lane);
#pragma unroll
        for (int j = 0; j < 8; ++j) ab[half * 8 + j] = __shfl_sync(0xffffffffu, sum, ((j & 1) << 4) | ((j >> 1 & 1) << 3) | ((j >> 2 & 1) << 2));
    }
    float U[GROUP][GROUP] = {}, O[GROUP][GROUP] = {};
#pragma unroll
    for (int t = 0; t < GROUP; ++t) {
        U[t][t] = __shfl_sync(0xffffffffu, beta, t);
#pragma unroll
        for (int s = 0; s < t; ++s) {
#pragma unroll
            for (int r = s; r < t; ++r) U[t][s] = fmaf(-U[t][t] * ab[t * (t - 1) / 2 + r], U[r][s], U[t][s]);
        }
#pragma unroll
        for (int s = 0; s <= t; ++s) {
#pragma unroll
            for (int r = s; r <= t; ++r) O[t][s] = fmaf(ab[6 + t * (t + 1) / 2 + r], U[r][s], O[t][s]);
        }
    }
    if (lane == 0) {
        float* scalars = rec + lay.scalars();
#pragma unroll
        for (int t = 0; t < GROUP; ++t) {
            st4_f32(scalars + t * GROUP, make_float4(U[t][0], U[t][1], U[t][2], U[t][3]));
            st4_f32(scalars + (GROUP + t) * GROUP, make_float4(O[t][0], O[t][1], O[t][2], O[t][3]));
        }
    }
    for (int c = lane * 4; c < p.dv; c += 128) {
        float4 v[GROUP];
        conv(p.v_off + h * p.dv + c, v);
#pragma unroll
        for (int t = 0; t < GROUP; ++t) st4_f32(rec + lay.values() + t * p.dv + c, v[t]);
    }
}

struct DeltaShape {
    int parts;               // CTAs that share a head's columns (a cluster)
    int cols;                // columns per CTA, whole consumer warps (the last part may reach past dv)
    int consumers;           // warps that run the recurrence
    int groups;              // groups per stage
};

template <class St>
__host__ __device__ constexpr RecordLayout layout_of() {
    return {St::DP, St::KQ_PITCH, St::KD_PITCH};
}

// The state of a warp's columns on the fp32 units: RGS row groups of RL rows (rows (j RGS + rg) 4 + e), 32 / RGS lanes side by side with
// CPT columns each; two rows packed.
template <int RGS, int RL, int CPT>
struct FmaState {
    static constexpr int DP = RGS * RL, LANES = 32 / RGS, COLS = LANES * CPT, KQ_PITCH = DP, KD_PITCH = DP, TEAM = 1, EXCHANGE = 0;
    static constexpr int MAX_WARPS = RL * CPT >= 64 ? 12 : 16;
    f32x2 S[RL / 2][CPT];
    int rg, col;             // row group, first column within the warp

    __device__ __forceinline__ int row_of(int i) const { return ((i >> 1) * RGS + rg) * 4 + (i & 1) * 2; }
    __device__ __forceinline__ void load(const float* state, int, int lane, int dk, int dv, bool has, float*) {
        rg = lane / LANES;
        col = lane % LANES * CPT;
#pragma unroll
        for (int i = 0; i < RL / 2; ++i)
#pragma unroll
            for (int c = 0; c < CPT; ++c) {
                const int r = row_of(i);
                const bool in = has && r < dk;
                S[i][c] = pack2(in ? state[(size_t)r * dv + col + c] : 0.f, in ? state[(size_t)(r + 1) * dv + col + c] : 0.f);
            }
    }
    __device__ __forceinline__ void store(float* state, int dk, int dv) const {
#pragma unroll
        for (int i = 0; i < RL / 2; ++i)
#pragma unroll
            for (int c = 0; c < CPT; ++c) {
                const int r = row_of(i);
                const float2 v = unpack2(S[i][c]);
                if (r < dk) {
                    state[(size_t)r * dv + col + c] = v.x;
                    state[(size_t)(r + 1) * dv + col + c] = v.y;
                }
            }
    }
    // st: staged record; sv, ys: its values and read-outs from this warp's first column on; sc: U and O
    __device__ __forceinline__ void group(const float* st, const float* sv, const float* sc, float* ys, int cols) {
        const RecordLayout lay = layout_of<FmaState>();
        const float* vec = st + rg * 4;
        f32x2 m2[GROUP][CPT], o2[GROUP][CPT];
#pragma unroll
        for (int t = 0; t < GROUP; ++t)
#pragma unroll
            for (int x = 0; x < CPT; ++x) m2[t][x] = o2[t][x] = 0ull;
#pragma unroll
        for (int j = 0; j < RL / 4; ++j) {
#pragma unroll
            for (int t = 0; t < GROUP; ++t) {
                const ulonglong2 kk = *reinterpret_cast<const ulonglong2*>(vec + t * DP + j * 4 * RGS);
                const ulonglong2 qq = *reinterpret_cast<const ulonglong2*>(vec + (GROUP + t) * DP + j * 4 * RGS);
#pragma unroll
                for (int x = 0; x < CPT; ++x) {
                    m2[t][x] = fma2(S[2 * j][x], kk.x, m2[t][x]);
                    m2[t][x] = fma2(S[2 * j + 1][x], kk.y, m2[t][x]);
                    o2[t][x] = fma2(S[2 * j][x], qq.x, o2[t][x]);
                    o2[t][x] = fma2(S[2 * j + 1][x], qq.y, o2[t][x]);
                }
            }
        }
        float u[CPT][GROUP];
#pragma unroll
        for (int x = 0; x < CPT; ++x) {
            float w[GROUP], o[GROUP];              // v - S^T c k, S^T c q
#pragma unroll
            for (int t = 0; t < GROUP; ++t) {
                const float2 ms = unpack2(m2[t][x]), os = unpack2(o2[t][x]);
                float m = ms.x + ms.y;
                o[t] = os.x + os.y;
#pragma unroll
                for (int d = LANES; d < 32; d *= 2) {
                    m += __shfl_xor_sync(0xffffffffu, m, d);
                    o[t] += __shfl_xor_sync(0xffffffffu, o[t], d);
                }
                w[t] = sv[t * cols + col + x] - m;
            }
            const float4 w4 = make_float4(w[0], w[1], w[2], w[3]);
#pragma unroll
            for (int t = 0; t < GROUP; ++t) {
                u[x][t] = dot4(ld4_f32(sc + t * GROUP), w4);
                if (rg == 0) ys[t * cols + col + x] = o[t] + dot4(ld4_f32(sc + (GROUP + t) * GROUP), w4);
            }
        }
#pragma unroll
        for (int j = 0; j < RL / 4; ++j) {
            const ulonglong2 gg = *reinterpret_cast<const ulonglong2*>(vec + lay.all() + j * 4 * RGS);
#pragma unroll
            for (int x = 0; x < CPT; ++x) {
                S[2 * j][x] = mul2(S[2 * j][x], gg.x);
                S[2 * j + 1][x] = mul2(S[2 * j + 1][x], gg.y);
            }
#pragma unroll
            for (int t = 0; t < GROUP; ++t) {
                const ulonglong2 kk = *reinterpret_cast<const ulonglong2*>(vec + lay.decayed() + t * DP + j * 4 * RGS);
#pragma unroll
                for (int x = 0; x < CPT; ++x) {
                    const f32x2 uu = pack2(u[x][t], u[x][t]);
                    S[2 * j][x] = fma2(kk.x, uu, S[2 * j][x]);
                    S[2 * j + 1][x] = fma2(kk.y, uu, S[2 * j + 1][x]);
                }
            }
        }
    }
};

// fp32 values as a sum of two tf32 values (the tensor core reads the upper 19 bits): three products of the parts give fp32 accuracy.
__device__ __forceinline__ void split(float v, uint32_t& hi, uint32_t& lo) {
    hi = __float_as_uint(v) & 0xffffe000u;
    lo = __float_as_uint(v - __uint_as_float(hi));
}
__device__ __forceinline__ void mma_k8(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void mma_k4(float (&d)[4], const uint32_t (&a)[2], uint32_t b) {
    asm("mma.sync.aligned.m16n8k4.row.col.f32.tf32.tf32.f32 {%0, %1, %2, %3}, {%4, %5}, {%6}, {%0, %1, %2, %3};"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(b));
}

// The state of 16 columns as accumulators of S^T (16 x DP, tiles of 8 rows of S), shared by a team of TEAM warps with ROWS rows each. The
// same registers are the first operand of S^T [c_t k_t | c_t q_t] - eight vectors, the width of a tile - because the order of the
// summation index is free: lane 4 r + i holds the rows 2 i and 2 i + 1 of a tile, which the product takes as its indices i and i + 4. Rows
// of S are dealt to tiles so that a lane's operands of four tiles lie together: tile 4 J + jj, row n is row 32 J + 4 n + jj of the warp's.
// The update S^T <- S^T c_4 + U^T [decayed k] has the four tokens as its summation index. The team adds up its sums over the rows through
// shared memory; all its warps then take the same steps.
template <int ROWS, int TEAM_>
struct MmaState {
    static constexpr int TEAM = TEAM_, DP = ROWS * TEAM, COLS = 16, KQ_PITCH = DP + 4, KD_PITCH = DP + 8;
    static constexpr int MAX_WARPS = ROWS >= 128 ? 12 : 16;
    static constexpr int EXCHANGE = TEAM > 1 ? 2 * 128 : 0;       // floats per warp
    float S[ROWS / 8][4];    // [tile]: (column r, row 2 i), (r, 2 i + 1), (r + 8, 2 i), (r + 8, 2 i + 1)
    float* sums;             // this team's exchange area, [2][TEAM][128]
    int r, i, member, team, flip;

    __device__ __forceinline__ int row_of(int tile, int n) const { return member * ROWS + (tile >> 2) * 32 + 4 * n + (tile & 3); }
    __device__ __forceinline__ void load(const float* state, int warp, int lane, int dk, int dv, bool has, float* exchange) {
        r = lane >> 2;
        i = lane & 3;
        team = warp / TEAM;
        member = warp % TEAM;
        sums = exchange + team * TEAM * EXCHANGE;
        flip = 0;
#pragma unroll
        for (int j = 0; j < ROWS / 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int row = row_of(j, 2 * i + (e & 1));
                S[j][e] = has && row < dk ? state[(size_t)row * dv + r + (e >> 1) * 8] : 0.f;
            }
    }
    __device__ __forceinline__ void store(float* state, int dk, int dv) const {
#pragma unroll
        for (int j = 0; j < ROWS / 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int row = row_of(j, 2 * i + (e & 1));
                if (row < dk) state[(size_t)row * dv + r + (e >> 1) * 8] = S[j][e];
            }
    }
    __device__ __forceinline__ void group(const float* st, const float* sv, const float* sc, float* ys, int cols) {
        const RecordLayout lay = layout_of<MmaState>();
        float acc[2][3][4] = {};                  // even and odd tiles, three products: independent chains
        const float* kq = st + r * KQ_PITCH + member * ROWS + 8 * i;      // vector r
#pragma unroll
        for (int J = 0; J < ROWS / 32; ++J) {
            const float4 f0 = ld4_f32(kq + J * 32), f1 = ld4_f32(kq + J * 32 + 4);
            const float b0[4] = {f0.x, f0.y, f0.z, f0.w}, b1[4] = {f1.x, f1.y, f1.z, f1.w};
#pragma unroll
            for (int jj = 0; jj < 4; ++jj) {
                const float (&t)[4] = S[4 * J + jj];
                uint32_t ah[4], al[4], h0, l0, h1, l1;
                split(t[0], ah[0], al[0]);
                split(t[2], ah[1], al[1]);
                split(t[1], ah[2], al[2]);
                split(t[3], ah[3], al[3]);
                split(b0[jj], h0, l0);
                split(b1[jj], h1, l1);
                mma_k8(acc[jj & 1][0], ah, h0, h1);
                mma_k8(acc[jj & 1][1], ah, l0, l1);
                mma_k8(acc[jj & 1][2], al, h0, h1);
            }
        }
        float z[4];                               // (column r, vectors 2 i and 2 i + 1), (column r + 8, ...): vectors 0..3 c k, 4..7 c q
#pragma unroll
        for (int e = 0; e < 4; ++e) z[e] = (acc[0][0][e] + acc[1][0][e]) + ((acc[0][1][e] + acc[1][1][e]) + (acc[0][2][e] + acc[1][2][e]));
        if constexpr (TEAM > 1) {                 // (two areas in turn: one barrier per group)
            float* area = sums + flip * TEAM * 128 + 16 * r + 4 * i;
            flip ^= 1;
            st4_f32(area + member * 128, make_float4(z[0], z[1], z[2], z[3]));
            asm volatile("bar.sync %0, %1;" ::"r"(team + 1), "n"(TEAM * 32) : "memory");
            z[0] = z[1] = z[2] = z[3] = 0.f;
#pragma unroll
            for (int m = 0; m < TEAM; ++m) {
                const float4 f = ld4_f32(area + m * 128);
                z[0] += f.x; z[1] += f.y; z[2] += f.z; z[3] += f.w;
            }
        }
        // lane i takes token i of the group: its row of U and of O, the step and the read-out of the columns r and r + 8
        const float4 row_u = ld4_f32(sc + i * GROUP), row_o = ld4_f32(sc + (GROUP + i) * GROUP);
        uint32_t uh[4], ul[2];
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            float w[GROUP];                       // v - S^T c k
#pragma unroll
            for (int t = 0; t < GROUP; ++t) w[t] = sv[t * cols + r + x * 8] - __shfl_sync(0xffffffffu, z[x * 2 + (t & 1)], (r << 2) | (t >> 1));
            const float even = __shfl_sync(0xffffffffu, z[x * 2], (r << 2) | 2 | (i >> 1)), odd = __shfl_sync(0xffffffffu, z[x * 2 + 1], (r << 2) | 2 | (i >> 1));
            const float4 w4 = make_float4(w[0], w[1], w[2], w[3]);
            if (TEAM == 1 || member == 0) ys[i * cols + r + x * 8] = (i & 1 ? odd : even) + dot4(row_o, w4);
            // u k in three products: high parts with both parts of k in one step of eight, low parts of u in one of four
            split(dot4(row_u, w4), uh[x], ul[x]);
            uh[x + 2] = uh[x];
        }
        const float* g = st + lay.all() + member * ROWS + 8 * i;
        const float* kd = st + lay.decayed() + i * KD_PITCH + member * ROWS + 4 * r;      // token i, rows 4 r ..
#pragma unroll
        for (int J = 0; J < ROWS / 32; ++J) {
            const float4 g0 = ld4_f32(g + J * 32), g1 = ld4_f32(g + J * 32 + 4), kk = ld4_f32(kd + J * 32);
            const float ga[4] = {g0.x, g0.y, g0.z, g0.w}, gb[4] = {g1.x, g1.y, g1.z, g1.w}, kf[4] = {kk.x, kk.y, kk.z, kk.w};
#pragma unroll
            for (int jj = 0; jj < 4; ++jj) {
                float (&t)[4] = S[4 * J + jj];
                t[0] *= ga[jj];
                t[2] *= ga[jj];
                t[1] *= gb[jj];
                t[3] *= gb[jj];
                uint32_t kh, kl;
                split(kf[jj], kh, kl);
                mma_k4(t, ul, kh);
                mma_k8(t, uh, kh, kl);
            }
        }
    }
};

template <class E, class St>
__global__ void __launch_bounds__(St::MAX_WARPS * 32, 1) delta_scan_kernel(ovb_delta_args p, DeltaShape s, int* status) {
    const RecordLayout lay = layout_of<St>();
    extern __shared__ __align__(16) float smem[];
    __shared__ uint64_t full[2];
    __shared__ volatile int abort_flag;
    const int group_len = lay.floats(s.cols), stage_len = s.groups * group_len, tokens = s.groups * GROUP;      // of a stage
    float* y_buf = smem + 2 * stage_len;           // [2][tokens][cols] read-outs
    float* s_norm = y_buf + 2 * tokens * s.cols;   // [cols], then the teams' exchange areas

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int part = blockIdx.x % s.parts, h = blockIdx.x / s.parts, b = blockIdx.y;
    const int c0 = part * s.cols, v_cols = max(0, min(s.cols, p.dv - c0));
    const bool consumer = warp < s.consumers;
    const int pw = warp - s.consumers, npw = (blockDim.x >> 5) - s.consumers;       // producer warps
    cg::cluster_group cluster = cg::this_cluster();
    auto barrier = [&]() {
        if (s.parts > 1) cluster.sync();
        else __syncthreads();
    };
    for (int i = threadIdx.x; i < s.cols; i += blockDim.x) s_norm[i] = c0 + i < p.dv ? p.norm[c0 + i] : 0.f;
    if (v_cols < s.cols) {                         // values that the copies leave out stay zero
        for (int i = threadIdx.x; i < 2 * stage_len; i += blockDim.x) smem[i] = 0.f;
        fence_proxy_async_smem();
    }
    if (threadIdx.x == 0) {
        abort_flag = 0;
        mbar_init(&full[0], 1);
        mbar_init(&full[1], 1);
        mbar_fence_init();
    }
    __syncthreads();
    pdl_enter();

    const int begin = p.subsequence_begins[b], len = p.subsequence_begins[b + 1] - begin, past = p.past_lens[b], slot = p.slots[b];
    const int groups = (len + GROUP - 1) / GROUP, stages = (groups + s.groups - 1) / s.groups;
    const int rec_len = lay.floats(p.dv);
    const float* records = p.records + ((size_t)first_group(p.subsequence_begins, b) * p.H + h) * rec_len;

    // one producer warp asks for the next stage: a bulk copy per record, or one and its part of the four rows of values
    auto fetch = [&](int c) {
        const int n = min(s.groups, groups - c * s.groups), head = s.parts > 1 ? lay.values() : rec_len, pieces = s.parts > 1 && v_cols > 0 ? 1 + GROUP : 1;
        uint64_t* bar = &full[c & 1];
        if (lane == 0) mbar_arrive_expect_tx(bar, n * (head + (pieces - 1) * v_cols) * 4);
        __syncwarp();
        for (int i = lane; i < n * pieces; i += 32) {
            const int g = i / pieces, x = i - g * pieces;
            const float* src = records + (size_t)(c * s.groups + g) * p.H * rec_len;
            float* dst = smem + (c & 1) * stage_len + g * group_len;
            if (x == 0) bulk_load_1d(dst, src, head * 4, bar);
            else bulk_load_1d(dst + lay.values() + (x - 1) * s.cols, src + lay.values() + (x - 1) * p.dv + c0, v_cols * 4, bar);
        }
    };
    auto landed = [&](int c) { mbar_wait(&full[c & 1], (c >> 1) & 1, &abort_flag, status); };      // (a wait that runs out shows in the status word)
    // norm, gate and store of the read-outs of stage c, up to four tokens of a warp side by side; columns of the other parts of the
    // cluster are read for the norm only
    auto finish = [&](int c) {
        constexpr int SIDE = 4;
        const int n = min(tokens, len - c * tokens), x = lane * 4;
        const float* ys = y_buf + (c & 1) * tokens * s.cols;
        const float* gate = p.low + (size_t)(begin + c * tokens) * p.ld_low + p.gate_off + (size_t)h * p.dv + c0;
        E* out = reinterpret_cast<E*>(p.out) + (size_t)(begin + c * tokens) * p.ldo + (size_t)h * p.o_head + c0;
        for (int first = pw; first < n; first += SIDE * npw) {
            float4 g[SIDE];
            float ss[SIDE];
#pragma unroll
            for (int i = 0; i < SIDE; ++i) {
                const int tt = first + i * npw;
                g[i] = tt < n && x < v_cols ? ld4_f32(gate + (size_t)tt * p.ld_low + x) : make_float4(0.f, 0.f, 0.f, 0.f);
                ss[i] = 0.f;
            }
            for (int col = x; col < s.parts * s.cols; col += 128) {
                const int from = s.parts > 1 ? col / s.cols : 0;
                const float* rows = ys + (col - from * s.cols);
                if (from != part) rows = cluster.map_shared_rank(rows, from);
#pragma unroll
                for (int i = 0; i < SIDE; ++i) {
                    const int tt = first + i * npw;
                    if (tt < n) {
                        const float4 y = ld4_f32(rows + tt * s.cols);
                        ss[i] += dot4(y, y);
                    }
                }
            }
#pragma unroll
            for (int d = 16; d > 0; d >>= 1)
#pragma unroll
                for (int i = 0; i < SIDE; ++i) ss[i] += __shfl_xor_sync(0xffffffffu, ss[i], d);
#pragma unroll
            for (int i = 0; i < SIDE; ++i) {
                const int tt = first + i * npw;
                if (tt >= n) break;
                const float inv = 1.f / sqrtf(ss[i] / (float)p.Dv + p.eps);
                for (int col = x; col < v_cols; col += 128) {
                    const float4 gv = col == x ? g[i] : ld4_f32(gate + (size_t)tt * p.ld_low + col);
                    st4_f32(out + (size_t)tt * p.ldo + col, mul4(scale4(mul4(ld4_f32(ys + tt * s.cols + col), ld4_f32(s_norm + col)), inv), sigmoid4<E>(gv)));
                }
            }
        }
    };

    St mine;
    const int cc = warp / St::TEAM * St::COLS;         // first column of a consumer warp
    float* state = p.state + ((size_t)slot * p.H + h) * p.dk * p.dv + c0 + cc;
    const bool inside = consumer && c0 + cc < p.dv;    // (dv is a multiple of 16: all columns of the warp or none)
    if (consumer) {
        mine.load(state, warp, lane, p.dk, p.dv, inside && past > 0, s_norm + s.cols);
    } else if (pw == 0) {
        fetch(0);
        landed(0);
    }
    barrier();
    for (int c = 0; c < stages; ++c) {
        if (consumer) {
            const int n = min(s.groups, groups - c * s.groups);
            for (int g = 0; g < n; ++g) {
                const float* st = smem + (c & 1) * stage_len + g * group_len;
                mine.group(st, st + lay.values() + cc, st + lay.scalars(), y_buf + ((c & 1) * tokens + g * GROUP) * s.cols + cc, s.cols);
            }
            fence_proxy_async_smem();              // (the next copies into this buffer come after these reads)
        } else {
            if (pw == 0 && c + 1 < stages) fetch(c + 1);
            if (c > 0) finish(c - 1);
            if (pw == 0 && c + 1 < stages) landed(c + 1);
        }
        barrier();
    }
    if (consumer) {
        if (inside) mine.store(state, p.dk, p.dv);
    } else {
        finish(stages - 1);
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

template <class E, int NV>
int launch_prepare(const ovb_delta_args& a, RecordLayout lay, cudaStream_t stream) {
    auto kern = a.taps == 1   ? delta_prepare_kernel<E, NV, 1>
                : a.taps == 2 ? delta_prepare_kernel<E, NV, 2>
                : a.taps == 3 ? delta_prepare_kernel<E, NV, 3>
                : a.taps == 4 ? delta_prepare_kernel<E, NV, 4>
                              : delta_prepare_kernel<E, NV, 0>;
    OVB_CHECK_CUDA(launch_pdl(kern, dim3(a.T / GROUP + a.B, ceil_div(a.H, 4)), dim3(128), 0, stream, a, lay));
    return 0;
}

template <class E, class St>
int launch_scan(const ovb_delta_args& a, int parts, cudaStream_t stream) {
    if (int rc = St::DP <= 128 ? launch_prepare<E, 1>(a, layout_of<St>(), stream) : launch_prepare<E, 2>(a, layout_of<St>(), stream)) return rc;
    constexpr int MAX_WARPS = St::MAX_WARPS;
    const int units = ceil_div(a.dv, St::COLS);
    while (parts < 8 && ceil_div(units, parts) * St::TEAM > MAX_WARPS - 2) parts *= 2;
    DeltaShape s;
    s.parts = parts;
    s.consumers = ceil_div(units, parts) * St::TEAM;
    if (s.consumers > MAX_WARPS - 2) {
        set_error("ovb_channel_delta: value size %d is too large", a.dv);
        return ERR_UNSUPPORTED;
    }
    s.cols = ceil_div(units, parts) * St::COLS;
    auto bytes = [&]() { return 4 * ((size_t)2 * s.groups * (layout_of<St>().floats(s.cols) + GROUP * s.cols) + s.cols + s.consumers * St::EXCHANGE); };
    s.groups = 8;
    while (s.groups > 1 && (bytes() > 226 * 1024 || s.groups * GROUP >= 2 * a.max_q_len)) s.groups /= 2;
    const size_t smem = bytes();
    OVB_REQUIRE(smem <= 226 * 1024, "ovb_channel_delta: heads of %d x %d need too much shared memory", a.dk, a.dv);
    const int most = s.parts > 1 ? 8 : 4, producers = MAX_WARPS - s.consumers < most ? MAX_WARPS - s.consumers : most;
    auto kern = delta_scan_kernel<E, St>;
    static std::atomic<uint64_t> configured{0};
    int dev = 0;
    OVB_CHECK_CUDA(cudaGetDevice(&dev));
    const uint64_t bit = 1ull << (dev & 63);
    if (!(configured.load(std::memory_order_acquire) & bit)) {
        OVB_CHECK_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024));
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
    OVB_CHECK_CUDA(cudaLaunchKernelEx(&cfg, kern, a, s, status_word()));
    return 0;
}

template <class E>
int launch_channel_delta(const ovb_delta_args& a, cudaStream_t stream) {
    OVB_REQUIRE(a.records && (reinterpret_cast<uintptr_t>(a.records) & 15) == 0, "ovb_channel_delta: no room for the groups' records");
    // one CTA per (sequence, head) when those fill the machine, else up to eight that share the columns
    int parts = 1;
    while (parts < 8 && a.B * a.H * parts * 2 <= 148 && a.dv >= 16 * parts * 2) parts *= 2;
    int rc;
    if constexpr (sizeof(E) == 2) {
        // (few sequences: teams share the rows as well)
        if (a.dk <= 32) rc = launch_scan<E, MmaState<32, 1>>(a, parts, stream);
        else if (a.dk <= 64) rc = parts > 1 ? launch_scan<E, MmaState<32, 2>>(a, parts, stream) : launch_scan<E, MmaState<64, 1>>(a, parts, stream);
        else if (a.dk <= 128) rc = parts > 1 ? launch_scan<E, MmaState<32, 4>>(a, parts, stream) : launch_scan<E, MmaState<128, 1>>(a, parts, stream);
        else rc = launch_scan<E, MmaState<64, 4>>(a, parts, stream);
    } else {
        rc = a.dk <= 32    ? launch_scan<E, FmaState<4, 8, 2>>(a, parts, stream)
             : a.dk <= 64  ? launch_scan<E, FmaState<4, 16, 2>>(a, parts, stream)
             : a.dk <= 128 ? launch_scan<E, FmaState<4, 32, 2>>(a, parts, stream)
                           : launch_scan<E, FmaState<8, 32, 2>>(a, parts, stream);
    }
    if (rc) return rc;
    return update_conv_ring<E>(a.proj, a.ldp, {a.conv_w, a.conv_ring, a.taps, a.conv_cols}, a.subsequence_begins, a.past_lens, a.slots, a.B, stream);
}

}  // namespace

}  // namespace ovb

extern "C" int64_t ovb_channel_delta_record_floats(int T, int B, int H, int dk, int dv) {
    // (the largest of the layouts: rows up to the next size that is served, vectors eight floats further apart)
    const int dp = dk <= 32 ? 32 : dk <= 64 ? 64 : dk <= 128 ? 128 : 256;
    return (int64_t)(T / ovb::GROUP + B) * H * ovb::RecordLayout{dp, dp + 8, dp + 8}.floats(dv);
}

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
        if (a->dk > 256) {
            set_error("ovb_channel_delta: key size %d above 256", a->dk);
            return ERR_UNSUPPORTED;
        }
        return launch_channel_delta<E>(*a, stream);
    });
}
