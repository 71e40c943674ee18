// From projections to what attention reads: per-head norms, rotary positions and the rows of the paged cache.
//
//   heads_prepare   grouped-query attention. Every query and key head may be RMS-normed over its dimensions (weights shared by
//                   the heads) and its first dimensions turned by the position; queries are changed in place, key and value
//                   rows go to the cache.
//   latent_prepare  latent attention. The low-rank row of a token is normed and cached together with the one turned key part
//                   that all heads share; the queries' turned part is written where the attention kernel reads it.
//
// A table of inverse frequencies (fp32, made by the host, whatever scaling it follows) and a multiplier of cos and sin describe
// the rotation; dimension i is paired with i + dims / 2. Norms, angles and sums are fp32. Rows of heads are padded to the pitch
// that the attention kernels want; the padding is zero and is never written.
#include "debug_bounds.cuh"
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

// Turn the pair (u, v) = (r[i], r[i + dims / 2]) of a row by pos * inv_freq[i].
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

struct HeadsParams {
    void* proj;              // [T, ldp]: query heads at column 0, key heads at k_off, value heads at v_off
    void* k_cache;           // [blocks, G, block_size, dk_pad]
    void* v_cache;           // [blocks, G, block_size, dv_pad]
    const float* q_norm;     // [D] or NULL
    const float* k_norm;
    const int* positions;
    const int* slot_map;
    Rotation rot;
    int T, H, G, D, Dv, dk_pad, dv_pad, ldp, k_off, v_off, block_size;
    float eps;
};

// One warp per (token, head); the row passes through shared memory because a rotation pairs elements of different lanes.
template <class E>
__global__ void __launch_bounds__(128) heads_prepare_kernel(HeadsParams p) {
    pdl_enter();
    extern __shared__ float rows[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t = blockIdx.x, head = blockIdx.y * 4 + warp;
    if (head >= p.H + 2 * p.G) return;
    E* proj = reinterpret_cast<E*>(p.proj) + (size_t)t * p.ldp;
    const bool is_q = head < p.H, is_k = !is_q && head < p.H + p.G;
    const int kvh = is_q ? 0 : (head - p.H) % p.G;
    E* src = is_q ? proj + head * p.dk_pad : is_k ? proj + p.k_off + kvh * p.dk_pad : proj + p.v_off + kvh * p.dv_pad;
    E* dst = src;
    if (!is_q) {
        const int slot = OVB_DBG_SLOT(p.slot_map[t], p.block_size);
        if (slot < 0) return;
        const size_t row = ((size_t)(slot / p.block_size) * p.G + kvh) * p.block_size + slot % p.block_size;
        dst = is_k ? reinterpret_cast<E*>(p.k_cache) + row * p.dk_pad : reinterpret_cast<E*>(p.v_cache) + row * p.dv_pad;
    }
    if (!is_q && !is_k) {
        for (int i = lane; i < p.Dv; i += 32) dst[i] = src[i];
        return;
    }
    float* r = rows + warp * p.D;
    float ss = 0.f;
    for (int i = lane; i < p.D; i += 32) {
        const float v = ld_f32(src + i);
        r[i] = v;
        ss += v * v;
    }
    const float* w = is_q ? p.q_norm : p.k_norm;
    if (w) {
        const float inv = 1.f / sqrtf(warp_sum(ss) / (float)p.D + p.eps);
        for (int i = lane; i < p.D; i += 32) r[i] *= inv * w[i];
    }
    __syncwarp();
    const int half = p.rot.dims / 2;
    const float pos = (float)p.positions[t];
    for (int i = lane; i < half; i += 32) turn(p.rot, pos, i, r[i], r[i + half]);
    __syncwarp();
    for (int i = lane; i < p.D; i += 32) st_f32(dst + i, r[i]);
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

int ovb_heads_prepare(const ovb_heads_args* a, ovb_stream_t stream) {
    OVB_REQUIRE(a && a->proj && a->k_cache && a->v_cache && a->positions && a->slot_map, "ovb_heads_prepare: null operand");
    OVB_REQUIRE(a->T > 0 && a->H > 0 && a->G > 0 && a->D > 0 && a->Dv > 0 && a->dk_pad >= a->D && a->dv_pad >= a->Dv && a->block_size > 0,
                "ovb_heads_prepare: bad sizes");
    OVB_REQUIRE(a->rot_dims >= 0 && a->rot_dims % 2 == 0 && a->rot_dims <= a->D && (a->rot_dims == 0 || a->inv_freq), "ovb_heads_prepare: bad rotation");
    OVB_REQUIRE(a->D <= 2048, "ovb_heads_prepare: head size %d above 2048", a->D);
    HeadsParams p = {a->proj, a->k_cache, a->v_cache, a->q_norm, a->k_norm, a->positions, a->slot_map, {a->inv_freq, a->rot_dims, a->rot_mult},
                     a->T, a->H, a->G, a->D, a->Dv, a->dk_pad, a->dv_pad, a->ldp, a->k_off, a->v_off, a->block_size, a->eps};
    return dispatch_store(a->dtype, "ovb_heads_prepare", [&](auto e) -> int {
        using E = decltype(e);
        OVB_CHECK_CUDA(launch_pdl(heads_prepare_kernel<E>, dim3(p.T, ceil_div(p.H + 2 * p.G, 4)), dim3(128), (size_t)4 * p.D * 4, (cudaStream_t)stream, p));
        return 0;
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
