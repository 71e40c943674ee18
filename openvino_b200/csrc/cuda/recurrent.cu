// Linear-recurrence layers of hybrid LLMs: the selective state-space scan (Mamba-2 form), the gated delta rule
// (Gated DeltaNet / Qwen3-Next linear attention) and, at the end of the file, the real-gated linear recurrent unit with its
// short convolution (Griffin's recurrent block). The first two walk the tokens of a sequence in order with the recurrent state
// of one head resident in registers: one warp owns four rows (state-space) or four columns (delta rule) of the state
// matrix, its 32 lanes hold the rows' elements, and the dot products of a token are warp shuffles (four sums share six
// shuffles). The state is read from and written to HBM once per launch; the token vectors every row of a head shares are
// staged in shared memory sixteen tokens at a time.
//
// Reference counterparts: the SelectiveSSM and GatedDeltaNet internal operations
// (src/common/transformations/include/ov_ops/, executed by the CPU plugin's recurrent kernels).
#include <stdlib.h>

#include <type_traits>

#include "common.cuh"
#include "sm100_ptx.cuh"
#include "store_types.cuh"
#include "warp_sums.cuh"

namespace ovb {

namespace {

constexpr int REC_WARPS = 8;     // warps per CTA
constexpr int REC_PER_WARP = 4;  // state rows (state-space) / columns (delta rule) per warp
constexpr int REC_TILE = REC_WARPS * REC_PER_WARP;   // rows / columns of one head per CTA
constexpr int REC_CHUNK = 16;    // tokens staged in shared memory at a time
constexpr int REC_MAXV = 8;      // state elements per lane: state widths up to 256

// state[b, h, p, :] <- state * exp(A[h] * dt) + dt * B[b, t, g, :] * x[b, t, h, p];  y[b, t, h, p] = <state, C[b, t, g, :]>
// One CTA owns RW * 8 rows p of one (b, h), each warp RW of them; the token vectors B, C (shared by all rows and by the
// heads of a group) are staged in shared memory REC_CHUNK tokens at a time, so that they cross L2 once per CTA and not
// once per row, and the outputs of a chunk leave through shared memory as whole rows of y.
template <int NV, int RW>
__global__ void __launch_bounds__(REC_WARPS * 32)
selective_ssm_kernel(const float* __restrict__ A, const float* __restrict__ dt, const float* __restrict__ Bm, const float* __restrict__ x,
                     const float* __restrict__ Cm, float* __restrict__ state, float* __restrict__ y, int L, int H, int P, int G, int S) {
    constexpr int TILE = REC_WARPS * RW;
    __shared__ float sB[REC_CHUNK][NV * 32], sC[REC_CHUNK][NV * 32], sX[REC_CHUNK][TILE], sY[REC_CHUNK][TILE], sD[REC_CHUNK], sDA[REC_CHUNK];
    const int bh = blockIdx.y, b = bh / H, h = bh % H, g = h / (H / G);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, p0 = blockIdx.x * TILE, pw = p0 + warp * RW;
    float st[RW][NV];
#pragma unroll
    for (int r = 0; r < RW; ++r)
#pragma unroll
        for (int i = 0; i < NV; ++i) st[r][i] = (pw + r < P && lane + 32 * i < S) ? state[((size_t)bh * P + pw + r) * S + lane + 32 * i] : 0.f;
    const float a = A[h];
    const int mine = RW == 8 ? rec_owned_value8(lane) : rec_owned_value(lane);
    const bool writer = RW == 8 ? (lane & 3) == 0 : (lane & 7) == 0;
    for (int t0 = 0; t0 < L; t0 += REC_CHUNK) {
        const int nt = min(REC_CHUNK, L - t0);
        const size_t tok0 = (size_t)b * L + t0;
        __syncthreads();
        for (int idx = threadIdx.x; idx < nt * NV * 32; idx += REC_WARPS * 32) {
            const int tt = idx / (NV * 32), s = idx % (NV * 32);
            sB[tt][s] = s < S ? Bm[((tok0 + tt) * G + g) * S + s] : 0.f;
            sC[tt][s] = s < S ? Cm[((tok0 + tt) * G + g) * S + s] : 0.f;
        }
        for (int idx = threadIdx.x; idx < nt * TILE; idx += REC_WARPS * 32) {
            const int tt = idx / TILE, r = idx % TILE;
            sX[tt][r] = p0 + r < P ? x[((tok0 + tt) * H + h) * P + p0 + r] : 0.f;
        }
        if (threadIdx.x < nt) {
            const float d = dt[(tok0 + threadIdx.x) * H + h];
            sD[threadIdx.x] = d;
            sDA[threadIdx.x] = expf(a * d);
        }
        __syncthreads();
#pragma unroll 2
        for (int tt = 0; tt < nt; ++tt) {
            const float d = sD[tt], dA = sDA[tt];
            float bv[NV], cv[NV], acc[RW];
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                bv[i] = sB[tt][lane + 32 * i] * d;
                cv[i] = sC[tt][lane + 32 * i];
            }
#pragma unroll
            for (int r = 0; r < RW; ++r) {
                const float xv = sX[tt][warp * RW + r];
                acc[r] = 0.f;
#pragma unroll
                for (int i = 0; i < NV; ++i) {
                    st[r][i] = st[r][i] * dA + bv[i] * xv;
                    acc[r] += st[r][i] * cv[i];
                }
            }
            float total;
            if constexpr (RW == 8) total = rec_reduce8(acc, lane);
            else total = rec_reduce4(acc[0], acc[1], acc[2], acc[3], lane);
            if (writer) sY[tt][warp * RW + mine] = total;
        }
        __syncthreads();
        for (int idx = threadIdx.x; idx < nt * TILE; idx += REC_WARPS * 32) {
            const int tt = idx / TILE, r = idx % TILE;
            if (p0 + r < P) y[((tok0 + tt) * H + h) * P + p0 + r] = sY[tt][r];
        }
    }
#pragma unroll
    for (int r = 0; r < RW; ++r)
#pragma unroll
        for (int i = 0; i < NV; ++i)
            if (pw + r < P && lane + 32 * i < S) state[((size_t)bh * P + pw + r) * S + lane + 32 * i] = st[r][i];
}

// Value columns iv of the state [Dk, Dv] of (b, hv):  S *= exp(g);  delta = (v - <S, k>) * beta;  S += k * delta;  y = <S, q>.
// q arrives scaled (and normalised where the layer asks for it), k normalised likewise. One CTA owns CW * 8 columns of one
// (b, hv), each warp CW of them; q and k of the head (shared by all its columns) are staged in shared memory REC_CHUNK
// tokens at a time, and the outputs of a chunk leave through shared memory as whole rows of y.
template <int NV, int CW>
__global__ void __launch_bounds__(REC_WARPS * 32)
gated_delta_rule_kernel(const float* __restrict__ q, const float* __restrict__ k, const float* __restrict__ v, const float* __restrict__ gate,
                        const float* __restrict__ beta, float* __restrict__ state, float* __restrict__ y, int L, int Hq, int Hv, int Dk, int Dv) {
    constexpr int TILE = REC_WARPS * CW;
    __shared__ float sQ[REC_CHUNK][NV * 32], sK[REC_CHUNK][NV * 32], sV[REC_CHUNK][TILE], sY[REC_CHUNK][TILE], sG[REC_CHUNK], sBt[REC_CHUNK];
    const int bh = blockIdx.y, b = bh / Hv, h = bh % Hv, hq = h / (Hv / Hq);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, c0 = blockIdx.x * TILE, cw = c0 + warp * CW;
    float st[CW][NV];
    float* sbase = state + (size_t)bh * Dk * Dv;
#pragma unroll
    for (int c = 0; c < CW; ++c)
#pragma unroll
        for (int i = 0; i < NV; ++i) st[c][i] = (cw + c < Dv && lane + 32 * i < Dk) ? sbase[(size_t)(lane + 32 * i) * Dv + cw + c] : 0.f;
    const int mine = CW == 8 ? rec_owned_value8(lane) : rec_owned_value(lane);
    const bool writer = CW == 8 ? (lane & 3) == 0 : (lane & 7) == 0;
    for (int t0 = 0; t0 < L; t0 += REC_CHUNK) {
        const int nt = min(REC_CHUNK, L - t0);
        const size_t tok0 = (size_t)b * L + t0;
        __syncthreads();
        for (int idx = threadIdx.x; idx < nt * NV * 32; idx += REC_WARPS * 32) {
            const int tt = idx / (NV * 32), d = idx % (NV * 32);
            sQ[tt][d] = d < Dk ? q[((tok0 + tt) * Hq + hq) * Dk + d] : 0.f;
            sK[tt][d] = d < Dk ? k[((tok0 + tt) * Hq + hq) * Dk + d] : 0.f;
        }
        for (int idx = threadIdx.x; idx < nt * TILE; idx += REC_WARPS * 32) {
            const int tt = idx / TILE, c = idx % TILE;
            sV[tt][c] = c0 + c < Dv ? v[((tok0 + tt) * Hv + h) * Dv + c0 + c] : 0.f;
        }
        if (threadIdx.x < nt) {
            sG[threadIdx.x] = expf(gate[(tok0 + threadIdx.x) * Hv + h]);
            sBt[threadIdx.x] = beta[(tok0 + threadIdx.x) * Hv + h];
        }
        __syncthreads();
        for (int tt = 0; tt < nt; ++tt) {
            const float decay = sG[tt], bt = sBt[tt];
            float kr[NV], qr[NV], mem[CW], o[CW];
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                kr[i] = sK[tt][lane + 32 * i];
                qr[i] = sQ[tt][lane + 32 * i];
            }
#pragma unroll
            for (int c = 0; c < CW; ++c) {
                mem[c] = 0.f;
#pragma unroll
                for (int i = 0; i < NV; ++i) {
                    st[c][i] *= decay;
                    mem[c] += st[c][i] * kr[i];
                }
            }
            float m;
            if constexpr (CW == 8) m = rec_reduce8(mem, lane);
            else m = rec_reduce4(mem[0], mem[1], mem[2], mem[3], lane);
#pragma unroll
            for (int c = 0; c < CW; ++c) {
                const int owner = CW == 8 ? (((c & 1) << 4) | (((c >> 1) & 1) << 3) | (((c >> 2) & 1) << 2)) : rec_owner_lane(c);
                const float delta = (sV[tt][warp * CW + c] - __shfl_sync(0xffffffffu, m, owner)) * bt;
                o[c] = 0.f;
#pragma unroll
                for (int i = 0; i < NV; ++i) {
                    st[c][i] += kr[i] * delta;
                    o[c] += st[c][i] * qr[i];
                }
            }
            float total;
            if constexpr (CW == 8) total = rec_reduce8(o, lane);
            else total = rec_reduce4(o[0], o[1], o[2], o[3], lane);
            if (writer) sY[tt][warp * CW + mine] = total;
        }
        __syncthreads();
        for (int idx = threadIdx.x; idx < nt * TILE; idx += REC_WARPS * 32) {
            const int tt = idx / TILE, c = idx % TILE;
            if (c0 + c < Dv) y[((tok0 + tt) * Hv + h) * Dv + c0 + c] = sY[tt][c];
        }
    }
#pragma unroll
    for (int c = 0; c < CW; ++c)
#pragma unroll
        for (int i = 0; i < NV; ++i)
            if (cw + c < Dv && lane + 32 * i < Dk) sbase[(size_t)(lane + 32 * i) * Dv + cw + c] = st[c][i];
}

// ------------------------------------------------------------------------------ real-gated linear recurrent unit
// Ragged batches: tokens subsequence_begins[b] .. of sequence b continue from the state in slot slots[b], or from zeros when
// past_lens[b] == 0 (a slot that another request used before needs no clearing). The state of a channel is S (fp32) and the
// last taps - 1 inputs of the convolution.

// u[t, c] = bias[c] + sum_j w[j, c] * x[t - (taps - 1) + j, c]. u is laid out block by block with a pitch of ub_pitch columns per
// block of bw channels, as the block-diagonal gate product reads it. A thread owns V consecutive channels of a strip of tokens.
template <int V>
__device__ __forceinline__ void conv_load(const float* src, float (&v)[V]) {
    if constexpr (V == 4) {
        const float4 q = ld4_f32(src);
        v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
    } else {
        v[0] = *src;
    }
}
template <int V>
__device__ __forceinline__ void conv_load(const __nv_bfloat16* src, float (&v)[V]) {
    if constexpr (V == 4) {
        const float4 q = ld4_f32(src);
        v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
    } else {
        v[0] = __bfloat162float(*src);
    }
}

constexpr int CONV_STRIP = 8;    // tokens per thread of a prompt

// TAPS > 0: the number of taps at compile time; a strip whose inputs all lie in one sequence's chunk then reads each of them once.
template <class E, int V, int TAPS>
__global__ void __launch_bounds__(128) causal_conv_kernel(ovb_rglru_args p, int strip) {
    pdl_enter();
    __shared__ int s_b;
    const int c = (blockIdx.y * 128 + threadIdx.x) * V, keep = p.taps - 1;
    int t = blockIdx.x * strip;
    const int t_end = min(p.T, t + strip);
    find_sequence(p.subsequence_begins, p.B, t, &s_b);
    __syncthreads();
    if (c >= p.N) return;
    int b = s_b;
    const E* x = reinterpret_cast<const E*>(p.x) + c;
    E* u = reinterpret_cast<E*>(p.u) + (c / p.bw) * p.ub_pitch + c % p.bw;
    auto put = [&](int tok, const float (&acc)[V]) {
        if constexpr (V == 4) st4_f32(u + (size_t)tok * p.ldu, make_float4(acc[0], acc[1], acc[2], acc[3]));
        else st_f32(u + (size_t)tok * p.ldu, acc[0]);
    };
    float bias[V];
    conv_load<V>(p.conv_b + c, bias);
    if (TAPS > 0 && strip == CONV_STRIP && t - (TAPS - 1) >= p.subsequence_begins[b] && t + CONV_STRIP <= p.subsequence_begins[b + 1]) {
        constexpr int KEEP = TAPS > 0 ? TAPS - 1 : 0, TW = TAPS > 0 ? TAPS : 1;
        float in[CONV_STRIP + KEEP][V], w[TW][V];
#pragma unroll
        for (int j = 0; j < CONV_STRIP + KEEP; ++j) conv_load<V>(x + (size_t)(t - KEEP + j) * p.ldx, in[j]);
#pragma unroll
        for (int j = 0; j < TW; ++j) conv_load<V>(p.conv_w + (size_t)j * p.N + c, w[j]);
#pragma unroll
        for (int k = 0; k < CONV_STRIP; ++k) {
            float acc[V];
#pragma unroll
            for (int i = 0; i < V; ++i) {
                acc[i] = bias[i];
#pragma unroll
                for (int j = 0; j < TW; ++j) acc[i] = fmaf(w[j][i], in[k + j][i], acc[i]);
            }
            put(t + k, acc);
        }
        return;
    }
    for (; t < t_end; ++t) {
        while (b + 1 < p.B && t >= p.subsequence_begins[b + 1]) ++b;
        const int begin = p.subsequence_begins[b];
        float acc[V];
#pragma unroll
        for (int i = 0; i < V; ++i) acc[i] = bias[i];
        for (int j = 0; j < p.taps; ++j) {
            const int s = t - keep + j;                  // token; before the chunk of the sequence: from its state
            float v[V] = {}, w[V];
            if (s >= begin) conv_load<V>(x + (size_t)s * p.ldx, v);
            else if (p.past_lens[b] != 0) conv_load<V>(p.conv_state + ((size_t)p.slots[b] * keep + s - begin + keep) * p.N + c, v);
            conv_load<V>(p.conv_w + (size_t)j * p.N + c, w);
#pragma unroll
            for (int i = 0; i < V; ++i) acc[i] = fmaf(w[i], v[i], acc[i]);
        }
        put(t, acc);
    }
}

__device__ __forceinline__ float rec_sigmoid(float z) { return __fdividef(1.f, 1.f + __expf(-z)); }
// gelu of the other branch: 0.5 z (1 + tanh(v)) = z * sigmoid(2 v)
__device__ __forceinline__ float rec_gelu_tanh(float z) { return z * rec_sigmoid(1.5957691216057308f * (z + 0.044715f * z * z * z)); }
__device__ __forceinline__ float rec_sqrt(float z) {
    float r;
    asm("sqrt.approx.f32 %0, %1;" : "=f"(r) : "f"(z));
    return r;
}

constexpr int LRU_PIECE = 8;    // tokens per warp and round of a prompt

// One group of 32 channels (a lane each) of one sequence. The NW warps of the group take consecutive pieces of LRU_L tokens: each
// composes the affine maps S -> a S + b of its piece, the pieces' maps are chained through shared memory, and the piece is then
// replayed from its true starting state. NW = 1 (decode): a CTA holds four independent groups.
template <class E, int NW, int LRU_L>
__global__ void __launch_bounds__(NW == 1 ? 128 : NW * 32, NW == 4 ? 7 : 1) lru_scan_kernel(ovb_rglru_args p) {
    pdl_enter();
    __shared__ float sA[2][NW][32], sB[2][NW][32];        // (two sets: one barrier per round)
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int b = blockIdx.y, w = NW == 1 ? 0 : warp;
    const int c = (NW == 1 ? blockIdx.x * 4 + warp : blockIdx.x) * 32 + lane;
    const bool live = c < p.N;
    const int begin = p.subsequence_begins[b], len = p.subsequence_begins[b + 1] - begin, slot = p.slots[b];
    const bool fresh = p.past_lens[b] == 0;
    const int cc = live ? c : 0, blk = cc / p.bw, cb = cc % p.bw;
    const float lam = p.log_decay[cc], br = p.gate_b[cc], bi = p.gate_b[p.N + cc];
    const float* gates = p.gates + (size_t)begin * p.ldg + blk * p.gb_pitch + cb;
    const E* us = reinterpret_cast<const E*>(p.u) + (size_t)begin * p.ldu + blk * p.ub_pitch + cb;
    const E* ys = reinterpret_cast<const E*>(p.y) + (size_t)begin * p.ldy + cc;
    E* out = reinterpret_cast<E*>(p.out) + (size_t)begin * p.ldo + cc;
    float* state = p.state + (size_t)slot * p.N + cc;
    float carry = fresh ? 0.f : *state;
    int set = 0;
    for (int t0 = 0; t0 < len; t0 += NW * LRU_L, set ^= 1) {
        const int tw = t0 + w * LRU_L, n = min(LRU_L, len - tw);
        float a[LRU_L], x[LRU_L], y[LRU_L], A = 1.f, S = 0.f;
        {
            float gr[LRU_L], gi[LRU_L];
#pragma unroll
            for (int k = 0; k < LRU_L; ++k) {             // all loads of the piece at once; past its end the last token again
                const size_t t = (size_t)min(tw + k, len - 1);
                gr[k] = gates[t * p.ldg];
                gi[k] = gates[t * p.ldg + p.gi_off];
                x[k] = ld_f32(us + t * p.ldu);
                y[k] = ld_f32(ys + t * p.ldy);
            }
#pragma unroll
            for (int k = 0; k < LRU_L; ++k) {
                // e = a - 1, exact for a close to one; 1 - a^2 = -e (2 + e)
                const float e = expm1f(-rec_sigmoid(gr[k] + br) * lam);
                a[k] = k < n ? 1.f + e : 1.f;
                x[k] = k < n ? rec_sqrt(-e * (2.f + e)) * rec_sigmoid(gi[k] + bi) * x[k] : 0.f;
                y[k] = rec_gelu_tanh(y[k]);
                S = fmaf(a[k], S, x[k]);
                A *= a[k];
            }
        }
        float s = carry;
        if (NW > 1) {
            sA[set][w][lane] = A;
            sB[set][w][lane] = S;
            __syncthreads();
#pragma unroll
            for (int k = 0; k < NW; ++k) {
                if (k == w) s = carry;
                carry = fmaf(sA[set][k][lane], carry, sB[set][k][lane]);
            }
        }
#pragma unroll
        for (int k = 0; k < LRU_L; ++k) {
            s = fmaf(a[k], s, x[k]);
            if (live && k < n) st_f32(out + (size_t)(tw + k) * p.ldo, s * y[k]);
        }
        if (NW == 1) carry = s;
    }
    if (!live || w != 0) return;
    *state = carry;
    const int keep = p.taps - 1;
    float* old = p.conv_state + (size_t)slot * keep * p.N + c;
    for (int j = 0; j < keep; ++j) {
        const int s = len - keep + j;                     // ascending j only reads rows that are not overwritten yet
        float v = 0.f;
        if (s >= 0) v = ld_f32(reinterpret_cast<const E*>(p.x) + (size_t)(begin + s) * p.ldx + c);
        else if (!fresh) v = old[(size_t)(s + keep) * p.N];
        old[(size_t)j * p.N] = v;
    }
}

// OVB_SSM_ROWS_PER_WARP = 4 keeps the four-row (four-column) form of both kernels for every shape (8 by default where it applies)
int env_rows_per_warp() {
    const char* e = getenv("OVB_SSM_ROWS_PER_WARP");
    return e && atoi(e) == 4 ? 4 : 8;
}

template <class Launch>
int dispatch_width(int width, Launch launch) {
    if (width <= 32) return launch(std::integral_constant<int, 1>());
    if (width <= 64) return launch(std::integral_constant<int, 2>());
    if (width <= 128) return launch(std::integral_constant<int, 4>());
    return launch(std::integral_constant<int, REC_MAXV>());
}

}  // namespace

}  // namespace ovb

extern "C" {

int ovb_selective_ssm(const float* A, const float* dt, const float* Bm, const float* x, const float* Cm, float* state, float* y, int B, int L, int H, int P,
                      int G, int S, ovb_stream_t stream_) {
    using namespace ovb;
    OVB_REQUIRE(A && dt && Bm && x && Cm && state && y, "ovb_selective_ssm: null argument");
    OVB_REQUIRE(B > 0 && L >= 0 && H > 0 && P > 0 && G > 0 && S > 0 && H % G == 0, "ovb_selective_ssm: bad sizes (heads %d, groups %d)", H, G);
    if (S > 32 * REC_MAXV) {
        set_error("ovb_selective_ssm: state size %d above %d", S, 32 * REC_MAXV);
        return ERR_UNSUPPORTED;
    }
    OVB_REQUIRE((long long)B * H <= 65535, "ovb_selective_ssm: batch x heads above 65535");
    cudaStream_t stream = (cudaStream_t)stream_;
    static const int rows_per_warp = env_rows_per_warp();
    return dispatch_width(S, [&](auto nv) -> int {
        constexpr int NV = decltype(nv)::value;
        // eight rows per warp halve the shared-memory reads and shuffles per row; they need 8 * NV state registers per lane
        if (NV <= 4 && P >= 64 && rows_per_warp == 8)
            selective_ssm_kernel<NV, 8><<<dim3(ceil_div(P, REC_WARPS * 8), B * H), REC_WARPS * 32, 0, stream>>>(A, dt, Bm, x, Cm, state, y, L, H, P, G, S);
        else
            selective_ssm_kernel<NV, 4><<<dim3(ceil_div(P, REC_WARPS * 4), B * H), REC_WARPS * 32, 0, stream>>>(A, dt, Bm, x, Cm, state, y, L, H, P, G, S);
        OVB_CHECK_CUDA(cudaGetLastError());
        return 0;
    });
}

int ovb_gated_delta_rule(const float* q, const float* k, const float* v, const float* gate, const float* beta, float* state, float* y, int B, int L, int Hq,
                         int Hv, int Dk, int Dv, ovb_stream_t stream_) {
    using namespace ovb;
    OVB_REQUIRE(q && k && v && gate && beta && state && y, "ovb_gated_delta_rule: null argument");
    OVB_REQUIRE(B > 0 && L >= 0 && Hq > 0 && Hv > 0 && Dk > 0 && Dv > 0 && Hv % Hq == 0, "ovb_gated_delta_rule: bad sizes (value heads %d, key heads %d)", Hv, Hq);
    if (Dk > 32 * REC_MAXV) {
        set_error("ovb_gated_delta_rule: key width %d above %d", Dk, 32 * REC_MAXV);
        return ERR_UNSUPPORTED;
    }
    OVB_REQUIRE((long long)B * Hv <= 65535, "ovb_gated_delta_rule: batch x value heads above 65535");
    cudaStream_t stream = (cudaStream_t)stream_;
    static const int cols_per_warp = env_rows_per_warp();
    return dispatch_width(Dk, [&](auto nv) -> int {
        constexpr int NV = decltype(nv)::value;
        if (NV <= 4 && Dv >= 64 && cols_per_warp == 8)
            gated_delta_rule_kernel<NV, 8><<<dim3(ceil_div(Dv, REC_WARPS * 8), B * Hv), REC_WARPS * 32, 0, stream>>>(q, k, v, gate, beta, state, y, L, Hq, Hv, Dk, Dv);
        else
            gated_delta_rule_kernel<NV, 4><<<dim3(ceil_div(Dv, REC_WARPS * 4), B * Hv), REC_WARPS * 32, 0, stream>>>(q, k, v, gate, beta, state, y, L, Hq, Hv, Dk, Dv);
        OVB_CHECK_CUDA(cudaGetLastError());
        return 0;
    });
}

static bool rec_aligned(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

static int check_rglru(const ovb_rglru_args* a, const char* what) {
    using namespace ovb;
    OVB_REQUIRE(a && a->x && a->u && a->conv_w && a->conv_b && a->subsequence_begins && a->past_lens && a->slots && a->conv_state, "%s: null operand", what);
    OVB_REQUIRE(a->B > 0 && a->B <= 65535 && a->T > 0 && a->N > 0 && a->taps > 0 && a->bw > 0 && a->N % a->bw == 0 && a->ub_pitch >= a->bw, "%s: bad sizes", what);
    return 0;
}

int ovb_causal_conv(const ovb_rglru_args* a, ovb_stream_t stream) {
    using namespace ovb;
    if (int rc = check_rglru(a, "ovb_causal_conv")) return rc;
    return dispatch_store(a->dtype, "ovb_causal_conv", [&](auto e) -> int {
        using E = decltype(e);
        const int strip = a->max_q_len <= 4 ? 1 : CONV_STRIP;      // (a new sequence for every token: no strip to walk)
        const bool vec = a->bw % 4 == 0 && a->ldx % 4 == 0 && a->ldu % 4 == 0 && a->ub_pitch % 4 == 0 && rec_aligned(a->x) && rec_aligned(a->u);
        const dim3 grid(ceil_div(a->T, strip), ceil_div(a->N, vec ? 512 : 128));
        auto go = [&](auto kern) -> int {
            OVB_CHECK_CUDA(launch_pdl(kern, grid, dim3(128), 0, (cudaStream_t)stream, *a, strip));
            return 0;
        };
        if (!vec) return go(causal_conv_kernel<E, 1, 0>);
        return a->taps == 2 ? go(causal_conv_kernel<E, 4, 2>) : a->taps == 3 ? go(causal_conv_kernel<E, 4, 3>) : a->taps == 4 ? go(causal_conv_kernel<E, 4, 4>)
                                                                                                             : go(causal_conv_kernel<E, 4, 0>);
    });
}

int ovb_lru_scan(const ovb_rglru_args* a, ovb_stream_t stream) {
    using namespace ovb;
    if (int rc = check_rglru(a, "ovb_lru_scan")) return rc;
    OVB_REQUIRE(a->y && a->gates && a->gate_b && a->log_decay && a->state && a->out, "ovb_lru_scan: null operand");
    return dispatch_store(a->dtype, "ovb_lru_scan", [&](auto e) -> int {
        using E = decltype(e);
        auto go = [&](auto kern, int channels, int threads) -> int {
            OVB_CHECK_CUDA(launch_pdl(kern, dim3(ceil_div(a->N, channels), a->B), dim3(threads), 0, (cudaStream_t)stream, *a));
            return 0;
        };
        if (a->max_q_len == 1) return go(lru_scan_kernel<E, 1, 1>, 128, 128);
        if (a->max_q_len <= LRU_PIECE) return go(lru_scan_kernel<E, 1, LRU_PIECE>, 128, 128);
        // many groups: small CTAs, several per SM; few groups: more warps on each sequence
        return (long long)ceil_div(a->N, 32) * a->B >= 4 * 148 ? go(lru_scan_kernel<E, 4, LRU_PIECE>, 32, 128)
                                                              : go(lru_scan_kernel<E, 16, LRU_PIECE>, 32, 512);
    });
}

}  // extern "C"
