// From projections to what attention reads: per-head norms, rotary positions and the rows of the paged cache.
//
//   heads_prepare   grouped-query attention. Every projected column may pass a short causal convolution; every query and key head
//                   may be RMS-normed over its dimensions (weights shared by the heads) and its first dimensions turned by the
//                   position; values may be mixed with those of an earlier layer. Queries are changed in place (or written to a
//                   buffer of their own when there is a convolution), key and value rows go to the cache.
//   latent_prepare  latent attention. The low-rank row of a token is normed and cached together with the one turned key part
//                   that all heads share; the queries' turned part is written where the attention kernel reads it.
//
// A table of inverse frequencies (fp32, made by the host, whatever scaling it follows) and a multiplier of cos and sin describe
// the rotation; heads_prepare takes the cosines and sines of the step's positions from a table (ovb_rope_table) that all layers share; dimension i is paired with i + dims / 2. Norms, angles and sums are fp32. Rows of heads are padded to the pitch
// that the attention kernels want; the padding is zero and is never written.
#include "debug_bounds.cuh"
#include "short_conv.cuh"
#include "sm100_ptx.cuh"
#include "store_types.cuh"

namespace ovb {

OVB_DEBUG_LIMITS_DEFINE

namespace {

struct Rotation {
    const float* inv_freq;   // [dims / 2]
    int dims;                // 0: no rotation
    float mult;
};

// Turn the pair (u, v) = (r[i], r[i + dims / 2]) of a row by pos * inv_freq[i], or by an angle of the table (cos, sin).
__device__ __forceinline__ void turn(const Rotation& rot, float pos, int i, float& u, float& v) {
    float s, c;
    sincosf(pos * rot.inv_freq[i], &s, &c);
    s *= rot.mult;
    c *= rot.mult;
    const float a = u * c - v * s, b = v * c + u * s;
    u = a;
    v = b;
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

__device__ __forceinline__ void turn_by(float2 cs, float& u, float& v) {
    const float a = u * cs.x - v * cs.y, b = v * cs.x + u * cs.y;
    u = a;
    v = b;
}

__global__ void rope_table_kernel(const int* __restrict__ positions, const float* __restrict__ inv_freq, float2* __restrict__ table, int n, int half, float mult) {
    pdl_enter();
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    float s, c;
    sincosf((float)positions[i / half] * inv_freq[i % half], &s, &c);
    table[i] = make_float2(c * mult, s * mult);
}

struct HeadUnit {            // what one warp works on: a query, key or value head
    bool is_q, is_k;
    int kvh, n, col;         // KV head, columns, first column in proj
};
__device__ __forceinline__ HeadUnit head_unit(const ovb_heads_args& p, int head) {
    HeadUnit u;
    u.is_q = head < p.H;
    u.is_k = !u.is_q && head < p.H + p.G;
    u.kvh = u.is_q ? 0 : (head - p.H) % p.G;
    u.n = u.is_q || u.is_k ? p.D : p.Dv;
    u.col = u.is_q ? head * p.dk_pad : u.is_k ? p.k_off + u.kvh * p.dk_pad : p.v_off + u.kvh * p.dv_pad;
    return u;
}
// Row of the paged cache (or of the query buffer) that takes token t of this head; NULL: no slot.
template <class E>
__device__ __forceinline__ E* head_row(const ovb_heads_args& p, const HeadUnit& u, int t) {
    if (u.is_q) return p.q_out ? reinterpret_cast<E*>(p.q_out) + (size_t)t * p.ldq + u.col : reinterpret_cast<E*>(p.proj) + (size_t)t * p.ldp + u.col;
    const int slot = OVB_DBG_SLOT(__ldg(p.slot_map + t), p.block_size);
    if (slot < 0) return nullptr;
    const size_t row = ((size_t)(slot / p.block_size) * p.G + u.kvh) * p.block_size + slot % p.block_size;
    return u.is_k ? reinterpret_cast<E*>(p.k_cache) + row * p.dk_pad : reinterpret_cast<E*>(p.v_cache) + row * p.dv_pad;
}

// One warp per (token, head); the row passes through shared memory because a rotation pairs elements of different lanes.
template <class E>
__global__ void __launch_bounds__(128) heads_prepare_kernel(ovb_heads_args p) {
    pdl_enter();
    extern __shared__ float rows[];
    __shared__ int s_b;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t = blockIdx.x, head = blockIdx.y * 4 + warp;
    if (p.taps > 0) {
        find_sequence(p.subsequence_begins, p.B, t, &s_b);
        __syncthreads();
    }
    if (head >= p.H + 2 * p.G) return;
    const HeadUnit u = head_unit(p, head);
    const E* src = reinterpret_cast<const E*>(p.proj) + u.col;
    E* dst = head_row<E>(p, u, t);
    float* r = rows + warp * max(p.D, p.Dv);
    const ShortConv cv = {p.conv_w, p.conv_ring, p.taps, p.conv_cols};
    float ss = 0.f;
    for (int i = lane; i < u.n; i += 32) {
        float v;
        if (p.taps > 0) {
            const int begin = p.subsequence_begins[s_b], pos = p.positions[t];
            float* ring = cv.ring + (size_t)p.slots[s_b] * cv.taps * cv.cols + u.col + i;
            v = 0.f;
            for (int j = 0; j < cv.taps; ++j)
                v = fmaf(cv.w[(size_t)j * cv.cols + u.col + i], conv_input(src + i, p.ldp, ring, cv, t, begin, pos, cv.taps - 1 - j), v);
            if (p.max_q_len == 1 && cv.taps > 1) ring[(size_t)(pos % cv.taps) * cv.cols] = ld_f32(src + (size_t)t * p.ldp + i);
        } else {
            v = ld_f32(src + (size_t)t * p.ldp + i);
        }
        r[i] = v;
        ss += v * v;
    }
    if (!u.is_q && !u.is_k) {
        E* first = p.v_mode ? reinterpret_cast<E*>(p.v_first) + (size_t)t * p.ld_vf + u.kvh * p.Dv : nullptr;
        for (int i = lane; i < u.n; i += 32) {
            float v = r[i];
            if (p.v_mode == 1) st_f32(first + i, v);
            if (p.v_mode == 2) v = (1.f - p.v_mix) * v + p.v_mix * ld_f32(first + i);
            if (dst) st_f32(dst + i, v);
        }
        return;
    }
    if (!dst) return;
    const float* w = u.is_q ? p.q_norm : p.k_norm;
    if (w) {
        const float inv = 1.f / sqrtf(warp_sum(ss) / (float)p.D + p.eps);
        for (int i = lane; i < p.D; i += 32) r[i] *= inv * w[i];
    }
    __syncwarp();
    const int half = p.rot_dims / 2;
    for (int i = lane; i < half; i += 32) turn_by(reinterpret_cast<const float2*>(p.rope)[(size_t)t * half + i], r[i], r[i + half]);
    __syncwarp();
    for (int i = lane; i < p.D; i += 32) st_f32(dst + i, r[i]);
}

constexpr int HEADS_STRIP = 16, HEADS_BATCH = 4;      // tokens per warp of a prompt, and of those in registers at a time

// The same for heads of up to 128 columns in pieces of four: a warp walks a strip of tokens of one head with its columns in registers
// (lane l: columns 4 l ..), so that every projected value is fetched once; rotation partners sit in other lanes. TAPS 0: no convolution.
template <class E, int TAPS>
__global__ void __launch_bounds__(128, sizeof(E) == 2 ? 7 : 4) heads_strip_kernel(ovb_heads_args p, int strip) {
    pdl_enter();
    __shared__ int s_b;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t0 = blockIdx.x * strip, t_end = min(p.T, t0 + strip), head = min(blockIdx.y * 4 + warp, p.H + 2 * p.G - 1);   // (the last head once more)
    constexpr int KEEP = TAPS > 1 ? TAPS - 1 : 0;
    const HeadUnit u = head_unit(p, head);
    const bool is_v = !u.is_q && !u.is_k;
    const int c = lane * 4;
    const bool live = c < u.n;
    const E* src = reinterpret_cast<const E*>(p.proj) + u.col + (live ? c : 0);
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    float4 w[TAPS > 0 ? TAPS : 1];
    float4 hist[KEEP > 0 ? KEEP : 1];
    if (TAPS > 0) {
#pragma unroll
        for (int j = 0; j < TAPS; ++j) w[j] = live ? ld4_f32(p.conv_w + (size_t)j * p.conv_cols + u.col + c) : zero;
    }
    const float* nw = u.is_q ? p.q_norm : u.is_k ? p.k_norm : nullptr;
    // the partner of column c is c + half (in the lower half) or c - half
    const int half = is_v ? 0 : p.rot_dims / 2;
    const bool lower = c < half, turned = c < 2 * half;
    const int partner = turned ? (lower ? lane + half / 4 : lane - half / 4) : lane;
    const ShortConv cv = {p.conv_w, p.conv_ring, TAPS, p.conv_cols};
    int b = 0, next = 0;                          // sequence, its end
    if (TAPS > 0) {
        find_sequence(p.subsequence_begins, p.B, t0, &s_b);
        __syncthreads();
        b = s_b;
        next = p.subsequence_begins[b + 1];
    }
    Raw4<E> ahead[HEADS_BATCH];
    auto request = [&](int tb) {
#pragma unroll
        for (int k = 0; k < HEADS_BATCH; ++k) {
            ahead[k].set(zero);
            if (live && tb + k < t_end) ahead[k].load(src + (size_t)(tb + k) * p.ldp);
        }
    };
    request(t0);
    for (int tb = t0; tb < t_end; tb += HEADS_BATCH) {
        Raw4<E> raw[HEADS_BATCH];
#pragma unroll
        for (int k = 0; k < HEADS_BATCH; ++k) raw[k] = ahead[k];
        request(tb + HEADS_BATCH);
#pragma unroll
        for (int k = 0; k < HEADS_BATCH; ++k) {
            const int t = tb + k;
            if (t >= t_end) break;
            float4 v = raw[k].get();
            if (TAPS > 0) {
                if (KEEP > 0 && (t == t0 || t >= next)) {      // what came before: this step's tokens, or the ring
                    while (t >= next) next = p.subsequence_begins[++b + 1];
                    const int begin = p.subsequence_begins[b], pos = p.positions[t];
                    float* ring = cv.ring + (size_t)p.slots[b] * TAPS * cv.cols + u.col + c;
#pragma unroll
                    for (int j = 0; j < KEEP; ++j) hist[j] = live ? conv_input4(src, p.ldp, ring, cv, t, begin, pos, KEEP - j) : zero;
                    if (p.max_q_len == 1 && live) st4_f32(ring + (size_t)(pos % TAPS) * cv.cols, v);
                }
                float4 acc = zero;
#pragma unroll
                for (int j = 0; j < KEEP; ++j) acc = fma4(w[j], hist[j], acc);
                acc = fma4(w[TAPS > 0 ? TAPS - 1 : 0], v, acc);
#pragma unroll
                for (int j = 0; j + 1 < KEEP; ++j) hist[j] = hist[j + 1];
                if (KEEP > 0) hist[KEEP - 1] = v;
                v = acc;
            }
            if (nw) {
                const float inv = 1.f / sqrtf(warp_sum(v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w) / (float)p.D + p.eps);
                if (live) v = make_float4(v.x * inv * __ldg(nw + c), v.y * inv * __ldg(nw + c + 1), v.z * inv * __ldg(nw + c + 2), v.w * inv * __ldg(nw + c + 3));
            }
            if (half > 0) {
                const float4 o = make_float4(__shfl_sync(0xffffffffu, v.x, partner), __shfl_sync(0xffffffffu, v.y, partner), __shfl_sync(0xffffffffu, v.z, partner),
                                             __shfl_sync(0xffffffffu, v.w, partner));
                if (turned) {
                    const float4* cs = reinterpret_cast<const float4*>(p.rope + ((size_t)t * half + (lower ? c : c - half)) * 2);
                    const float4 a = __ldg(cs), d = __ldg(cs + 1);       // (cos, sin) of four pairs
                    const float sg = lower ? -1.f : 1.f;     // lower: u cos - v sin, upper: v cos + u sin
                    v = make_float4(v.x * a.x + sg * (o.x * a.y), v.y * a.z + sg * (o.y * a.w), v.z * d.x + sg * (o.z * d.y), v.w * d.z + sg * (o.w * d.w));
                }
            }
            if (is_v && p.v_mode && live) {
                E* first = reinterpret_cast<E*>(p.v_first) + (size_t)t * p.ld_vf + u.kvh * p.Dv + c;
                if (p.v_mode == 1) {
                    st4_f32(first, v);
                } else {
                    const float4 f = ld4_f32(first);
                    const float a = 1.f - p.v_mix;
                    v = make_float4(a * v.x + p.v_mix * f.x, a * v.y + p.v_mix * f.y, a * v.z + p.v_mix * f.z, a * v.w + p.v_mix * f.w);
                }
            }
            E* dst = head_row<E>(p, u, t);
            if (dst && live) st4_f32(dst + c, v);
        }
    }
}

struct LatentParams {
    void* proj;              // [T, ldp]: H query heads of q_pitch columns (unrotated part, then the turned part at q_rot_off),
                             // the low-rank row at c_off, the shared key part at kr_off
    void* q_rot;             // turned query parts go here: + t * ld_qr + head * qr_pitch
    void* cache;             // [blocks, block_size, row_pitch]: low-rank row at 0, shared key part at key_off
    const float* c_norm;     // [C]
    const int* positions;
    const int* slot_map;
    Rotation rot;
    int T, H, C, R, q_pitch, q_rot_off, c_off, kr_off, ldp, ld_qr, qr_pitch, row_pitch, key_off, block_size;
    float eps;
};

// One CTA per token: warp 0 norms and caches the low-rank row and the shared key part, the other warps turn the query heads.
template <class E>
__global__ void __launch_bounds__(256) latent_prepare_kernel(LatentParams p) {
    pdl_enter();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t = blockIdx.x, half = p.rot.dims / 2;
    const float pos = (float)p.positions[t];
    E* proj = reinterpret_cast<E*>(p.proj) + (size_t)t * p.ldp;
    if (warp == 0) {
        const int slot = OVB_DBG_SLOT(p.slot_map[t], p.block_size);
        if (slot < 0) return;
        E* row = reinterpret_cast<E*>(p.cache) + (size_t)slot * p.row_pitch;
        const E* c = proj + p.c_off;
        const int nvec = p.C / 4;             // (rows and offsets are multiples of 16 elements)
        float ss = 0.f;
#pragma unroll 4
        for (int i = lane; i < nvec; i += 32) {
            const float4 v = ld4_f32(c + i * 4);
            ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
        for (int i = nvec * 4 + lane; i < p.C; i += 32) ss += ld_f32(c + i) * ld_f32(c + i);
        const float inv = 1.f / sqrtf(warp_sum(ss) / (float)p.C + p.eps);
#pragma unroll 4
        for (int i = lane; i < nvec; i += 32) {
            const float4 v = ld4_f32(c + i * 4), g = ld4_f32(p.c_norm + i * 4);
            st4_f32(row + i * 4, make_float4(v.x * inv * g.x, v.y * inv * g.y, v.z * inv * g.z, v.w * inv * g.w));
        }
        for (int i = nvec * 4 + lane; i < p.C; i += 32) st_f32(row + i, ld_f32(c + i) * inv * p.c_norm[i]);
        const E* kr = proj + p.kr_off;
        for (int i = lane; i < half; i += 32) {
            float u = ld_f32(kr + i), v = ld_f32(kr + i + half);
            turn(p.rot, pos, i, u, v);
            st_f32(row + p.key_off + i, u);
            st_f32(row + p.key_off + i + half, v);
        }
        for (int i = p.rot.dims + lane; i < p.R; i += 32) row[p.key_off + i] = kr[i];
        return;
    }
    for (int idx = (warp - 1) * 32 + lane; idx < p.H * half; idx += 224) {
        const int h = idx / half, i = idx % half;
        const E* q = proj + h * p.q_pitch + p.q_rot_off;
        E* dst = reinterpret_cast<E*>(p.q_rot) + (size_t)t * p.ld_qr + h * p.qr_pitch;
        float u = ld_f32(q + i), v = ld_f32(q + i + half);
        turn(p.rot, pos, i, u, v);
        st_f32(dst + i, u);
        st_f32(dst + i + half, v);
    }
    for (int idx = (warp - 1) * 32 + lane; idx < p.H * (p.R - p.rot.dims); idx += 224) {
        const int h = idx / (p.R - p.rot.dims), i = p.rot.dims + idx % (p.R - p.rot.dims);
        reinterpret_cast<E*>(p.q_rot)[(size_t)t * p.ld_qr + h * p.qr_pitch + i] = proj[h * p.q_pitch + p.q_rot_off + i];
    }
}

}  // namespace

}  // namespace ovb

#ifdef OVB_DEBUG_BOUNDS
extern "C" int ovb_debug_set_limits_heads(const ovb::DebugLimits* l) {
    OVB_CHECK_CUDA(cudaMemcpyToSymbol(ovb::g_dbg_limits, l, sizeof(*l)));
    return 0;
}
#endif

extern "C" {
using namespace ovb;

int ovb_rope_table(const int* positions, const float* inv_freq, float* table, int T, int half, float mult, ovb_stream_t stream) {
    OVB_REQUIRE(positions && inv_freq && table && T > 0 && half > 0, "ovb_rope_table: bad arguments");
    OVB_CHECK_CUDA(launch_pdl(rope_table_kernel, dim3(ceil_div(T * half, 256)), dim3(256), 0, (cudaStream_t)stream, positions, inv_freq,
                              reinterpret_cast<float2*>(table), T * half, half, mult));
    return 0;
}

int ovb_heads_prepare(const ovb_heads_args* a, ovb_stream_t stream) {
    OVB_REQUIRE(a && a->proj && a->k_cache && a->v_cache && a->positions && a->slot_map, "ovb_heads_prepare: null operand");
    OVB_REQUIRE(a->T > 0 && a->H > 0 && a->G > 0 && a->D > 0 && a->Dv > 0 && a->dk_pad >= a->D && a->dv_pad >= a->Dv && a->block_size > 0,
                "ovb_heads_prepare: bad sizes");
    OVB_REQUIRE(a->rot_dims >= 0 && a->rot_dims % 2 == 0 && a->rot_dims <= a->D && (a->rot_dims == 0 || a->rope), "ovb_heads_prepare: bad rotation");
    OVB_REQUIRE(a->D <= 2048 && a->Dv <= 2048, "ovb_heads_prepare: head sizes %d, %d above 2048", a->D, a->Dv);
    OVB_REQUIRE(a->taps == 0 || (a->taps > 0 && a->conv_w && a->conv_ring && a->subsequence_begins && a->past_lens && a->slots && a->q_out && a->B > 0 &&
                                 a->conv_cols >= a->v_off + a->G * a->dv_pad), "ovb_heads_prepare: bad short convolution");
    OVB_REQUIRE(a->v_mode == 0 || (a->v_first && a->ld_vf >= a->G * a->Dv && (a->v_mode == 1 || a->v_mode == 2)), "ovb_heads_prepare: bad value mixing");
    auto aligned = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
    const int units = a->H + 2 * a->G;
    // heads in registers: whole pieces of four columns everywhere, rotation partners at whole lanes
    const bool strip_form = a->D <= 128 && a->Dv <= 128 && a->D % 4 == 0 && a->Dv % 4 == 0 && a->rot_dims % 8 == 0 && a->taps <= 4 &&
                            a->ldp % 4 == 0 && a->dk_pad % 4 == 0 && a->dv_pad % 4 == 0 && a->k_off % 4 == 0 && a->v_off % 4 == 0 && a->conv_cols % 4 == 0 &&
                            a->ldq % 4 == 0 && a->ld_vf % 4 == 0 && aligned(a->proj) && aligned(a->q_out) && aligned(a->k_cache) && aligned(a->v_cache) &&
                            aligned(a->conv_w) && aligned(a->conv_ring) && aligned(a->v_first) && aligned(a->rope);
    return dispatch_store(a->dtype, "ovb_heads_prepare", [&](auto e) -> int {
        using E = decltype(e);
        if (strip_form) {
            // few tokens: a warp each; many: strips that share the inputs of the convolution
            const int strip = (long long)a->T * units <= 148 * 32 || a->max_q_len == 1 ? 1 : HEADS_STRIP;
            auto kern = a->taps == 0   ? heads_strip_kernel<E, 0>
                        : a->taps == 1 ? heads_strip_kernel<E, 1>
                        : a->taps == 2 ? heads_strip_kernel<E, 2>
                        : a->taps == 3 ? heads_strip_kernel<E, 3>
                                       : heads_strip_kernel<E, 4>;
            OVB_CHECK_CUDA(launch_pdl(kern, dim3(ceil_div(a->T, strip), ceil_div(units, 4)), dim3(128), 0, (cudaStream_t)stream, *a, strip));
        } else {
            const int width = a->D > a->Dv ? a->D : a->Dv;
            OVB_CHECK_CUDA(launch_pdl(heads_prepare_kernel<E>, dim3(a->T, ceil_div(units, 4)), dim3(128), (size_t)4 * width * 4, (cudaStream_t)stream, *a));
        }
        // (a decode step's kernel has written the ring itself)
        if (a->taps == 0 || a->max_q_len == 1) return 0;
        return update_conv_ring<E>(a->proj, a->ldp, {a->conv_w, a->conv_ring, a->taps, a->conv_cols}, a->subsequence_begins, a->past_lens, a->slots, a->B,
                                   (cudaStream_t)stream);
    });
}

int ovb_latent_prepare(const ovb_latent_args* a, ovb_stream_t stream) {
    OVB_REQUIRE(a && a->proj && a->q_rot && a->cache && a->c_norm && a->positions && a->slot_map, "ovb_latent_prepare: null operand");
    OVB_REQUIRE(a->T > 0 && a->H > 0 && a->C > 0 && a->R > 0 && a->block_size > 0 && a->key_off >= a->C && a->key_off + a->R <= a->row_pitch,
                "ovb_latent_prepare: bad sizes");
    OVB_REQUIRE(a->rot_dims > 0 && a->rot_dims % 2 == 0 && a->rot_dims <= a->R && a->inv_freq, "ovb_latent_prepare: bad rotation");
    OVB_REQUIRE(a->ldp % 4 == 0 && a->c_off % 4 == 0 && a->row_pitch % 4 == 0 && (reinterpret_cast<uintptr_t>(a->c_norm) & 15) == 0,
                "ovb_latent_prepare: rows must be aligned to 4 elements");
    LatentParams p = {a->proj, a->q_rot, a->cache, a->c_norm, a->positions, a->slot_map, {a->inv_freq, a->rot_dims, a->rot_mult},
                      a->T, a->H, a->C, a->R, a->q_pitch, a->q_rot_off, a->c_off, a->kr_off, a->ldp, a->ld_qr, a->qr_pitch, a->row_pitch, a->key_off,
                      a->block_size, a->eps};
    return dispatch_store(a->dtype, "ovb_latent_prepare", [&](auto e) -> int {
        using E = decltype(e);
        OVB_CHECK_CUDA(launch_pdl(latent_prepare_kernel<E>, dim3(p.T), dim3(256), 0, (cudaStream_t)stream, p));
        return 0;
    });
}

}  // extern "C"
