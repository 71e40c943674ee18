// Latent attention in its absorbed form, and the expansion of cached rows for prefill.
//
// latent_attention_kernel: every query head attends to the same cached row per token; the first part of that row is also the value.
// One CTA serves one token (decode: one sequence), 16 or 32 of its heads and one share of the visible keys. Key tiles of 64 rows
// pass through two shared-memory stages (cp.async), once for both products:
//   scores   warp w multiplies the heads' queries with keys 8w .. 8w + 7 of the tile,
//   softmax  running maximum over the CTA (per-warp maxima through shared memory), P as bf16 in shared memory,
//   sums     warp w owns its own slice of the value columns for all 64 keys, so the accumulator needs no merge.
// With split keys the partial sums go to scratch and the decode kernels' merge finishes.
//
// latent_gather_kernel: the rows that the windows of a batch's new tokens reach, made contiguous, so that a plain product expands
// them to per-head keys and values for the tcgen05 prefill kernel.
#include <math_constants.h>

#include <atomic>

#include "attention.cuh"
#include "common.cuh"
#include "debug_bounds.cuh"
#include "mma_sync.cuh"

namespace ovb {

OVB_DEBUG_LIMITS_DEFINE

namespace {

constexpr int kWarps = 8, kKeys = 64;

struct LatentKParams {
    PaKParams p;
    int row, pitch, cpad;     // elements of a cached row that take part, its pitch in shared memory (whole 128 bytes), value columns
};

__device__ __forceinline__ uint32_t row_off(int r, int chunk, int pitch) { return uint32_t(r * pitch * 2 + ((chunk ^ (r & 7)) << 4)); }

template <int MT, int VT>
__global__ void __launch_bounds__(kWarps * 32, 1) latent_attention_kernel(LatentKParams a) {
    pdl_enter_attn();
    const PaKParams& p = a.p;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 127) & ~uintptr_t(127));
    const int pitch = a.pitch, nch = a.row / 8, ksteps = a.row / 16;
    const int stage = kKeys * pitch * 2;
    uint8_t* sQ = smem;
    uint8_t* sK = sQ + MT * 16 * pitch * 2;                              // two stages
    uint8_t* sP = sK + 2 * stage;                                        // [MT * 16][64] bf16
    float* sMax = reinterpret_cast<float*>(sP + MT * 16 * kKeys * 2);    // [MT * 16][8]
    __shared__ int s_b;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t = blockIdx.x, h0 = blockIdx.y * MT * 16, split = blockIdx.z;
    if (threadIdx.x == 0) {
        int b = 0;
        while (b + 1 < p.B && t >= p.subsequence_begins[b + 1]) ++b;
        s_b = b;
    }
    for (int r = warp; r < MT * 16; r += kWarps) {
        const bool valid = h0 + r < p.Hq;
        const uint8_t* src = reinterpret_cast<const uint8_t*>(p.q) + ((size_t)t * p.ldq + (size_t)(valid ? h0 + r : 0) * p.q_head) * 2;
        for (int c = lane; c < nch; c += 32) cp_async16(sQ + row_off(r, c, pitch), src + c * 16, valid);
    }
    __syncthreads();
    const int b = s_b;
    const int ctx = p.past_lens[b] + t - p.subsequence_begins[b] + 1;    // keys that exist for this token
    const int lo = p.sliding_window > 0 ? max(0, ctx - p.sliding_window) : 0;
    const int k_lo = lo / kKeys * kKeys + split * p.keys_per_split;
    const int k_hi = min(ctx, k_lo + p.keys_per_split);
    const int ntiles = k_hi > k_lo ? (k_hi - k_lo + kKeys - 1) / kKeys : 0;
    const int* blocks = p.block_indices + p.block_indices_begins[b];
    auto load = [&](int tile, int st) {
        const int j0 = k_lo + tile * kKeys + warp * 8;                   // a warp's eight rows lie in one page
        const bool any = j0 < k_hi;
        const int blk = any ? OVB_DBG_BLOCK(blocks[j0 / p.block_size]) : 0;
        const uint8_t* src = reinterpret_cast<const uint8_t*>(p.k_cache) + ((size_t)blk * p.block_size + (any ? j0 % p.block_size : 0)) * p.k_row * 2;
        uint8_t* dst = sK + st * stage;
#pragma unroll
        for (int r = 0; r < 8; ++r)
            for (int c = lane; c < nch; c += 32) cp_async16(dst + row_off(warp * 8 + r, c, pitch), src + ((size_t)r * p.k_row) * 2 + c * 16, j0 + r < k_hi);
    };
    if (ntiles > 0) load(0, 0);
    cp_async_commit();

    float o[MT][VT * 2][4];
    float m_run[MT][2], l_run[MT][2];
#pragma unroll
    for (int m = 0; m < MT; ++m) {
#pragma unroll
        for (int i = 0; i < VT * 2; ++i) o[m][i][0] = o[m][i][1] = o[m][i][2] = o[m][i][3] = 0.f;
        m_run[m][0] = m_run[m][1] = -CUDART_INF_F;
        l_run[m][0] = l_run[m][1] = 0.f;
    }
    for (int tile = 0; tile < ntiles; ++tile) {
        const int st = tile & 1;
        cp_async_wait<0>();
        __syncthreads();                                                 // the tile has landed; the other stage and sP are free
        if (tile + 1 < ntiles) load(tile + 1, st ^ 1);
        cp_async_commit();
        const uint8_t* kS = sK + st * stage;
        // ---- scores of keys 8 * warp .. + 7 (two accumulators: even and odd steps)
        float s[MT][2][4];
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int i = 0; i < 4; ++i) s[m][0][i] = s[m][1][i] = 0.f;
#pragma unroll 2
        for (int ks = 0; ks < ksteps; ks += 2) {
            uint32_t k0, k1, k2, k3;
            ldsm_x4(smem_u32(kS + row_off(warp * 8 + (lane & 7), ks * 2 + (lane >> 3), pitch)), k0, k1, k2, k3);
#pragma unroll
            for (int m = 0; m < MT; ++m) {
                uint32_t q[4];
                const int r = m * 16 + (lane & 7) + 8 * ((lane >> 3) & 1);
                ldsm_x4(smem_u32(sQ + row_off(r, ks * 2 + (lane >> 4), pitch)), q[0], q[1], q[2], q[3]);
                mma16816<false>(s[m][0], q, k0, k1);
                if (ks + 1 < ksteps) {
                    ldsm_x4(smem_u32(sQ + row_off(r, ks * 2 + 2 + (lane >> 4), pitch)), q[0], q[1], q[2], q[3]);
                    mma16816<false>(s[m][1], q, k2, k3);
                }
            }
        }
        // ---- mask, maximum over the tile
        const int j = k_lo + tile * kKeys + warp * 8 + (lane & 3) * 2;
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int ri = 0; ri < 2; ++ri) {
                float mx = -CUDART_INF_F;
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const bool ok = j + e >= lo && j + e < k_hi;
                    const float v = ok ? (s[m][0][ri * 2 + e] + s[m][1][ri * 2 + e]) * p.scale_log2 : -CUDART_INF_F;
                    s[m][0][ri * 2 + e] = v;
                    mx = fmaxf(mx, v);
                }
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
                if ((lane & 3) == 0) sMax[(m * 16 + ri * 8 + (lane >> 2)) * kWarps + warp] = mx;
            }
        __syncthreads();
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int ri = 0; ri < 2; ++ri) {
                const int r = m * 16 + ri * 8 + (lane >> 2);
                const float4 x = *reinterpret_cast<const float4*>(sMax + r * kWarps), y = *reinterpret_cast<const float4*>(sMax + r * kWarps + 4);
                const float mnew = fmaxf(m_run[m][ri], fmaxf(fmaxf(fmaxf(x.x, x.y), fmaxf(x.z, x.w)), fmaxf(fmaxf(y.x, y.y), fmaxf(y.z, y.w))));
                const float base = mnew == -CUDART_INF_F ? 0.f : mnew;
                const float corr = exp2f(m_run[m][ri] - base);
                const float e0 = exp2f(s[m][0][ri * 2] - base), e1 = exp2f(s[m][0][ri * 2 + 1] - base);
                m_run[m][ri] = mnew;
                l_run[m][ri] = l_run[m][ri] * corr + e0 + e1;
                *reinterpret_cast<uint32_t*>(sP + row_off(r, warp, kKeys) + (lane & 3) * 4) = pack_bf16x2(e0, e1);
#pragma unroll
                for (int i = 0; i < VT * 2; ++i) {
                    o[m][i][ri * 2] *= corr;
                    o[m][i][ri * 2 + 1] *= corr;
                }
            }
        __syncthreads();
        // ---- O += P V for this warp's value columns
#pragma unroll
        for (int kk = 0; kk < kKeys / 16; ++kk) {
            uint32_t pf[MT][4];
#pragma unroll
            for (int m = 0; m < MT; ++m)
                ldsm_x4(smem_u32(sP + row_off(m * 16 + (lane & 7) + 8 * ((lane >> 3) & 1), kk * 2 + (lane >> 4), kKeys)), pf[m][0], pf[m][1], pf[m][2], pf[m][3]);
#pragma unroll
            for (int v = 0; v < VT; ++v) {
                const int col = (warp * VT + v) * 16;
                if (col >= a.cpad) break;
                uint32_t b0, b1, b2, b3;
                const int q = lane >> 3;
                ldsm_x4_t(smem_u32(kS + row_off(kk * 16 + (q & 1) * 8 + (lane & 7), col / 8 + (q >> 1), pitch)), b0, b1, b2, b3);
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    mma16816<false>(o[m][2 * v], pf[m], b0, b1);
                    mma16816<false>(o[m][2 * v + 1], pf[m], b2, b3);
                }
            }
        }
    }
    cp_async_wait<0>();
    // ---- denominators: every warp holds the sums over its own keys
    __syncthreads();
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int ri = 0; ri < 2; ++ri) {
            float l = l_run[m][ri];
            l += __shfl_xor_sync(0xffffffffu, l, 1);
            l += __shfl_xor_sync(0xffffffffu, l, 2);
            if ((lane & 3) == 0) sMax[(m * 16 + ri * 8 + (lane >> 2)) * kWarps + warp] = l;
        }
    __syncthreads();
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int ri = 0; ri < 2; ++ri) {
            const int r = m * 16 + ri * 8 + (lane >> 2), h = h0 + r;
            if (h >= p.Hq) continue;
            float l = 0.f;
#pragma unroll
            for (int w = 0; w < kWarps; ++w) l += sMax[r * kWarps + w];
            const float inv = p.nsplit > 1 ? 1.f : (l > 0.f ? 1.f / l : 0.f);
            float* sc = p.scratch + (((size_t)t * p.Hq + h) * p.nsplit + split) * (a.cpad + 2);
#pragma unroll
            for (int i = 0; i < VT * 2; ++i) {
                const int col = warp * VT * 16 + i * 8 + (lane & 3) * 2;
                if (col >= a.cpad) break;
                if (p.nsplit > 1) {
                    sc[col] = o[m][i][ri * 2];
                    sc[col + 1] = o[m][i][ri * 2 + 1];
                } else {
                    *reinterpret_cast<uint32_t*>(reinterpret_cast<__nv_bfloat16*>(p.out) + (size_t)t * p.ldo + (size_t)h * p.o_head + col) =
                        pack_bf16x2(o[m][i][ri * 2] * inv, o[m][i][ri * 2 + 1] * inv);
                }
            }
            if (p.nsplit > 1 && warp == 0 && (lane & 3) == 0) {
                sc[a.cpad] = m_run[m][ri];
                sc[a.cpad + 1] = l;
            }
        }
}

template <int MT, int VT>
int launch_latent(const LatentKParams& a, cudaStream_t stream) {
    const int smem = (MT * 16 + 2 * kKeys) * a.pitch * 2 + MT * 16 * kKeys * 2 + MT * 16 * kWarps * 4 + 128;
    if (smem > 227 * 1024 - 64) return ERR_UNSUPPORTED;
    auto kern = latent_attention_kernel<MT, VT>;
    static std::atomic<uint64_t> configured{0};   // one bit per device; raised to the whole limit once
    int dev = 0;
    OVB_CHECK_CUDA(cudaGetDevice(&dev));
    const uint64_t bit = 1ull << (dev & 63);
    if (!(configured.load(std::memory_order_acquire) & bit)) {
        OVB_CHECK_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024 - 64));
        configured.fetch_or(bit, std::memory_order_release);
    }
    OVB_CHECK_CUDA(launch_pdl(kern, dim3(a.p.T, ceil_div(a.p.Hq, MT * 16), a.p.nsplit), dim3(kWarps * 32), (size_t)smem, stream, a));
    return a.p.nsplit > 1 ? launch_decode_combine(a.p, a.cpad, stream) : 0;
}

__global__ void __launch_bounds__(256) latent_gather_kernel(const uint8_t* __restrict__ cache, uint8_t* __restrict__ out, int* __restrict__ kv_rows,
                                                            const int* __restrict__ past_lens, const int* __restrict__ subsequence_begins,
                                                            const int* __restrict__ block_indices, const int* __restrict__ block_indices_begins, int B, int rows,
                                                            int bytes, int row_bytes, int out_bytes, int window, int block_size) {
    pdl_enter();
    extern __shared__ int s_begin[];         // [B + 1] first gathered row of every sequence
    if (threadIdx.x < 32) {
        int carry = 0;
        for (int b0 = 0; b0 < B; b0 += 32) {
            const int b = b0 + threadIdx.x;
            int n = 0;
            if (b < B) n = past_lens[b] + subsequence_begins[b + 1] - subsequence_begins[b] - latent_first_key(past_lens[b], window);
            int incl = n;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int v = __shfl_up_sync(0xffffffffu, incl, o);
                if ((int)threadIdx.x >= o) incl += v;
            }
            if (b < B) s_begin[b] = carry + incl - n;
            carry += __shfl_sync(0xffffffffu, incl, 31);
        }
        if (threadIdx.x == 0) s_begin[B] = carry;
    }
    __syncthreads();
    if (blockIdx.x == 0)
        for (int b = threadIdx.x; b <= B; b += 256) kv_rows[b] = s_begin[b];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int r = blockIdx.x * 64 + warp; r < min(rows, (int)blockIdx.x * 64 + 64); r += 8) {
        int lo = 0, hi = B;                  // last b with s_begin[b] <= r
        while (lo + 1 < hi) {
            const int mid = (lo + hi) / 2;
            if (s_begin[mid] <= r) lo = mid;
            else hi = mid;
        }
        if (r >= s_begin[B]) break;
        const int j = latent_first_key(past_lens[lo], window) + r - s_begin[lo];
        const int blk = OVB_DBG_BLOCK(block_indices[block_indices_begins[lo] + j / block_size]);
        const uint8_t* src = cache + ((size_t)blk * block_size + j % block_size) * row_bytes;
        for (int c = lane * 16; c < bytes; c += 512) *reinterpret_cast<uint4*>(out + (size_t)r * out_bytes + c) = *reinterpret_cast<const uint4*>(src + c);
    }
}

}  // namespace

int launch_latent_attention(PaKParams p, int row, int cpad, int max_q_len, int max_ctx, long long scratch_bytes, cudaStream_t stream) {
    if (p.block_size % 8 || row % 16 || cpad > 512 || row > 1024 || p.k_row % 8 || p.ldq % 8 || p.q_head % 8 || p.ldo % 2 || p.o_head % 2 ||
        (reinterpret_cast<uintptr_t>(p.q) & 15) || (reinterpret_cast<uintptr_t>(p.k_cache) & 15) || (reinterpret_cast<uintptr_t>(p.out) & 3) || p.T > (1 << 30))
        return ERR_UNSUPPORTED;
    LatentKParams a;
    a.p = p;
    a.row = row;
    a.pitch = (row + 63) / 64 * 64;
    a.cpad = cpad;
    a.p.dv_store = cpad;
    const int mt = p.Hq <= 16 ? 1 : 2;
    const int keys = p.sliding_window > 0 && p.sliding_window + kKeys - 1 < max_ctx ? p.sliding_window + kKeys - 1 : max_ctx;
    const int tiles = ceil_div(keys, kKeys), ctas = p.T * ceil_div(p.Hq, mt * 16);
    int best = 1;
    if (max_q_len == 1 && p.T == p.B && p.scratch != nullptr) {
        // shares of the keys: whole waves of one CTA per SM, a fixed cost of about two key tiles per CTA and one for the merge
        double best_cost = 1e30;
        for (int n = 1; n <= 32 && n <= tiles; ++n) {
            if ((long long)ctas * 16 * mt * n * (cpad + 2) * 4 > scratch_bytes) break;
            const double cost = ceil_div(ctas * n, 148) * (ceil_div(tiles, n) + 2.0) + (n > 1 ? 1.0 : 0.0);
            if (cost < best_cost) {
                best_cost = cost;
                best = n;
            }
        }
    }
    a.p.nsplit = best;
    a.p.keys_per_split = ceil_div(tiles, best) * kKeys;
    const int vt = cpad <= 128 ? 1 : cpad <= 256 ? 2 : 4;
    if (mt == 1) return vt == 1 ? launch_latent<1, 1>(a, stream) : vt == 2 ? launch_latent<1, 2>(a, stream) : launch_latent<1, 4>(a, stream);
    return vt == 1 ? launch_latent<2, 1>(a, stream) : vt == 2 ? launch_latent<2, 2>(a, stream) : launch_latent<2, 4>(a, stream);
}

}  // namespace ovb

#ifdef OVB_DEBUG_BOUNDS
extern "C" int ovb_debug_set_limits_latent(const ovb::DebugLimits* l) {
    OVB_CHECK_CUDA(cudaMemcpyToSymbol(ovb::g_dbg_limits, l, sizeof(*l)));
    return 0;
}
#endif

extern "C" {
using namespace ovb;

int ovb_latent_gather(const void* cache, void* out, int* kv_rows, const int* past_lens, const int* subsequence_begins, const int* block_indices,
                      const int* block_indices_begins, int B, int rows, int cols, int row_pitch, int out_pitch, int window, int block_size, ovb_stream_t stream) {
    OVB_REQUIRE(cache && out && kv_rows && past_lens && subsequence_begins && block_indices && block_indices_begins && B > 0 && B <= 8192 && rows > 0,
                "ovb_latent_gather: bad arguments");
    OVB_REQUIRE(cols % 8 == 0 && row_pitch % 8 == 0 && out_pitch % 8 == 0 && cols <= row_pitch && cols <= out_pitch,
                "ovb_latent_gather: rows must be multiples of 8 elements");
    OVB_CHECK_CUDA(launch_pdl(latent_gather_kernel, dim3(ceil_div(rows, 64)), dim3(256), (size_t)(B + 1) * 4, (cudaStream_t)stream, (const uint8_t*)cache,
                              (uint8_t*)out, kv_rows, past_lens, subsequence_begins, block_indices, block_indices_begins, B, rows, cols * 2, row_pitch * 2,
                              out_pitch * 2, window, block_size));
    return 0;
}

int ovb_latent_prefill(const ovb_latent_prefill_args* a, ovb_stream_t stream) {
    OVB_REQUIRE(a && a->q && a->kv && a->cache && a->out && a->kv_rows && a->past_lens && a->subsequence_begins && a->block_indices && a->block_indices_begins,
                "ovb_latent_prefill: null operand");
    OVB_REQUIRE(a->B > 0 && a->T > 0 && a->H > 0 && a->rows > 0 && a->scale > 0.f, "ovb_latent_prefill: bad sizes");
    PaKParams p;
    memset(&p, 0, sizeof(p));
    p.q = a->q;
    p.out = a->out;
    p.k_cache = a->kv;
    p.v_cache = reinterpret_cast<const uint8_t*>(a->kv) + (size_t)a->v_off * 2;
    p.past_lens = a->past_lens;
    p.subsequence_begins = a->subsequence_begins;
    p.block_indices = a->block_indices;
    p.block_indices_begins = a->block_indices_begins;
    p.B = a->B; p.T = a->T; p.Hq = p.Hkv = a->H; p.group = 1;
    p.ldq = a->ldq; p.q_head = a->q_head; p.ldo = a->ldo; p.o_head = a->o_head;
    p.k_row = p.v_row = 8;                     // (pages hold the shared part only)
    p.kv_rows = a->kv_rows; p.kv_total = a->rows; p.kv_ld = a->ld_kv; p.k_head = a->k_head; p.v_head = a->v_head;
    p.shared = a->cache; p.shared_row = a->row_pitch; p.shared_col = a->key_off; p.q_shared = a->q_rot_off;
    p.block_size = a->block_size; p.sliding_window = a->window; p.causal = 1;
    p.scale_log2 = a->scale * 1.4426950408889634f;
    const int rc = launch_window_tc(p, a->k_head, a->R, a->Dv, (cudaStream_t)stream);
    if (rc == ERR_UNSUPPORTED) set_error("ovb_latent_prefill: sizes %d + %d / %d are not served", a->k_head, a->R, a->Dv);
    return rc;
}

}  // extern "C"
