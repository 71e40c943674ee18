// Latent attention in its absorbed form, and the expansion of cached rows for prefill.
//
// latent_attention_kernel: every query head attends to the same cached row per token; the first part of that row is also the value.
// One CTA of four warps serves one token (decode: one sequence), 16 of its heads and one share of the visible keys; several CTAs
// share an SM and hide each other's barriers. Key tiles of 16 rows pass through three shared-memory stages, one bulk copy per page,
// and are read for both products:
//   scores   the warps split the row's columns in quarters; the queries' fragments of a warp's quarter stay in registers for the
//            whole loop. The four partial sums meet in shared memory.
//   softmax  8 neighbouring threads per head add the partials, mask, keep running maximum and sum; P as bf16. The maximum is only
//            raised when a tile exceeds it by more than a factor of 2^8, so the accumulators are rarely rescaled.
//   sums     every warp owns its own slice of the value columns for all keys of the tile, so the accumulator needs no merge.
// The products of a step are the scores of tile t + 1 and the sums of tile t: independent, between the same two barriers.
// Pages keep the cache's row pitch in shared memory: a pitch of an odd number of 16-byte pieces spreads ldmatrix over all banks.
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

constexpr int kWarps = 4, kKeys = 16, kHeads = 16, kStages = 3;
constexpr int kScorePitch = kKeys + 8;    // floats per row of partial scores
constexpr int kPPitch = 48;               // bytes per row of P

struct LatentKParams {
    PaKParams p;
    int row, cpad;            // elements of a cached row that take part, value columns (multiples of 16)
    int block_shift;          // log2 of the block size
    int* status;
};

// A thread's reads of a stage are done before a bulk copy that is issued after the next barrier may write it. (ldmatrix results that
// are only needed later may otherwise still be outstanding: seen as wrong queries when they shared the first stage to be refilled.)
__device__ __forceinline__ void fence_reads_before_copies() { asm volatile("fence.proxy.async.shared::cta;" ::: "memory"); }

// VT: 16-column pieces of the value per warp; KQ: most 16-column steps in a quarter of the row; FULL: row and value fill them exactly.
template <int VT, int KQ, bool FULL>
__global__ void __launch_bounds__(kWarps * 32, 3) latent_attention_kernel(LatentKParams a) {
    constexpr int R = kHeads, TPR = kWarps * 32 / R;                     // rows, threads per row (two keys each)
    static_assert(TPR * 2 == kKeys, "softmax threads cover the tile");
    const PaKParams& p = a.p;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 127) & ~uintptr_t(127));
    const int pitch = p.k_row * 2, ksteps = a.row / 16;
    const int stage = kKeys * pitch;
    uint8_t* sK = smem;
    uint8_t* sQ = sK + 2 * stage;                                        // queries pass through the last stage
    float* sS = reinterpret_cast<float*>(sK + kStages * stage);          // partial scores [4][R][kScorePitch]
    uint8_t* sP = reinterpret_cast<uint8_t*>(sS + 4 * R * kScorePitch);
    float* sCorr = reinterpret_cast<float*>(sP + R * kPPitch);           // [R]
    float* sMax = sCorr + R;                                             // [R]
    uint64_t* full = reinterpret_cast<uint64_t*>(sMax + R);              // [kStages]
    volatile int* abort_flag = reinterpret_cast<volatile int*>(full + kStages);
    int* s_b = const_cast<int*>(abort_flag) + 1;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int t = blockIdx.x, h0 = blockIdx.y * R, split = blockIdx.z;
    if (tid == 0) {
        for (int i = 0; i < kStages; ++i) mbar_init(&full[i], 1);
        mbar_fence_init();
        *abort_flag = 0;
    }
    pdl_enter_attn();
    find_sequence(p.subsequence_begins, p.B, t, s_b);
    for (int r = warp; r < R; r += kWarps) {
        const bool valid = h0 + r < p.Hq;
        const uint8_t* src = reinterpret_cast<const uint8_t*>(p.q) + ((size_t)t * p.ldq + (size_t)(valid ? h0 + r : 0) * p.q_head) * 2;
        for (int c = lane; c < a.row / 8; c += 32) cp_async16(sQ + r * pitch + c * 16, src + c * 16, valid);
    }
    cp_async_commit();
    __syncthreads();
    const int b = *s_b;
    const int ctx = p.past_lens[b] + t - p.subsequence_begins[b] + 1;    // keys that exist for this token
    const int lo = p.sliding_window > 0 ? max(0, ctx - p.sliding_window) : 0;
    const int k_lo = lo / kKeys * kKeys + split * p.keys_per_split;
    const int k_hi = min(ctx, k_lo + p.keys_per_split);
    const int ntiles = k_hi > k_lo ? (k_hi - k_lo + kKeys - 1) / kKeys : 0;
    const int* blocks = p.block_indices + p.block_indices_begins[b];
    // One lane of warp 0 copies each page (or the tile's part of it); its place is looked up a tile ahead. Rows of a page past the
    // last key hold what the cache holds there: finite, and masked.
    const int seg = min(p.block_size, kKeys), nseg = kKeys / seg;
    const uint8_t* next_part = nullptr;
    auto look_up = [&](int tile) {
        if (warp == 0 && lane < nseg && tile < ntiles) {
            int j = k_lo + tile * kKeys + lane * seg;
            if (j >= k_hi) j = (k_hi - 1) / seg * seg;                   // (pages shorter than a tile: the last one again)
            const int blk = OVB_DBG_BLOCK(blocks[j >> a.block_shift]);
            next_part = reinterpret_cast<const uint8_t*>(p.k_cache) + (((size_t)blk << a.block_shift) + (j & (p.block_size - 1))) * pitch;
        }
    };
    auto load = [&](int tile) {
        if (warp == 0 && tile < ntiles) {
            const int st = tile % kStages;
            if (lane == 0) mbar_arrive_expect_tx(&full[st], stage);
            if (lane < nseg) bulk_load_1d(sK + st * stage + lane * seg * pitch, next_part, seg * pitch, &full[st]);
        }
        look_up(tile + 1);
    };
    look_up(0);
    load(0);
    load(1);
    cp_async_wait<0>();
    __syncthreads();
    // ---- this warp's quarter of the queries, in registers
    const int per = FULL ? KQ : (ksteps + 3) / 4, k0 = warp * per, kn = FULL ? KQ : max(0, min(per, ksteps - k0));
    uint32_t qf[KQ][4];
#pragma unroll
    for (int i = 0; i < KQ; ++i) {
        const int ks = FULL ? k0 + i : min(k0 + min(i, max(kn - 1, 0)), ksteps - 1);     // (steps past the end are not used)
        ldsm_x4(smem_u32(sQ + ((lane & 7) + 8 * ((lane >> 3) & 1)) * pitch + ks * 32 + (lane >> 4) * 16), qf[i][0], qf[i][1], qf[i][2], qf[i][3]);
    }
    float o[VT * 2][4];
#pragma unroll
    for (int i = 0; i < VT * 2; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    const int srow = tid / TPR, sc = tid % TPR;                          // softmax: this thread's row and place in it
    float m_run = -CUDART_INF_F, l_run = 0.f;
    bool ok = true;
    fence_reads_before_copies();
    __syncthreads();                                                     // the queries are out of the last stage
    load(2);
    const int gm = lane >> 3;
    const uint32_t k_off = ((gm >> 1) * 8 + (lane & 7)) * pitch + k0 * 32 + (gm & 1) * 16;               // score operand of step 0
    const uint32_t v_off = ((gm & 1) * 8 + (lane & 7)) * pitch + warp * (VT * 32) + (gm >> 1) * 16;      // value operand of piece 0
    for (int tile = -1; tile < ntiles; ++tile) {
        // ---- products: scores of tile + 1, sums of tile
        const bool more = tile + 1 < ntiles;
        if (more) ok = mbar_wait(&full[(tile + 1) % kStages], ((tile + 1) / kStages) & 1, abort_flag, a.status);
        const uint32_t kS = smem_u32(sK + (more ? (tile + 1) % kStages : 0) * stage) + k_off;
        const uint32_t vS = smem_u32(sK + (tile < 0 ? 0 : tile % kStages) * stage) + v_off;
        uint32_t pf[4];
        if (tile >= 0) {
            const float c0 = sCorr[lane >> 2], c1 = sCorr[8 + (lane >> 2)];
            ldsm_x4(smem_u32(sP + ((lane & 7) + 8 * ((lane >> 3) & 1)) * kPPitch + (lane >> 4) * 16), pf[0], pf[1], pf[2], pf[3]);
            if (__any_sync(0xffffffffu, c0 != 1.f || c1 != 1.f)) {
#pragma unroll
                for (int i = 0; i < VT * 2; ++i) {
                    o[i][0] *= c0; o[i][1] *= c0;
                    o[i][2] *= c1; o[i][3] *= c1;
                }
            }
        }
        float s[2][4];
#pragma unroll
        for (int n = 0; n < 2; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
        if (FULL && more && tile >= 0) {
#pragma unroll
            for (int i = 0; i < (KQ > VT ? KQ : VT); ++i) {
                uint32_t f[4], g[4];
                if (i < KQ) ldsm_x4(kS + i * 32, f[0], f[1], f[2], f[3]);
                if (i < VT) ldsm_x4_t(vS + i * 32, g[0], g[1], g[2], g[3]);
                if (i < KQ) {
                    mma16816<false>(s[0], qf[i], f[0], f[1]);
                    mma16816<false>(s[1], qf[i], f[2], f[3]);
                }
                if (i < VT) {
                    mma16816<false>(o[2 * i], pf, g[0], g[1]);
                    mma16816<false>(o[2 * i + 1], pf, g[2], g[3]);
                }
            }
        } else {
            if (more) {
#pragma unroll
                for (int i = 0; i < KQ; ++i)
                    if (i < kn) {
                        uint32_t f[4];
                        ldsm_x4(kS + i * 32, f[0], f[1], f[2], f[3]);
                        mma16816<false>(s[0], qf[i], f[0], f[1]);
                        mma16816<false>(s[1], qf[i], f[2], f[3]);
                    }
            }
            if (tile >= 0) {
#pragma unroll
                for (int w = 0; w < VT; ++w)
                    if ((warp * VT + w) * 16 < a.cpad) {
                        uint32_t g[4];
                        ldsm_x4_t(vS + w * 32, g[0], g[1], g[2], g[3]);
                        mma16816<false>(o[2 * w], pf, g[0], g[1]);
                        mma16816<false>(o[2 * w + 1], pf, g[2], g[3]);
                    }
            }
        }
        if (!more) break;
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int ri = 0; ri < 2; ++ri)
                *reinterpret_cast<float2*>(sS + (warp * R + ri * 8 + (lane >> 2)) * kScorePitch + n * 8 + (lane & 3) * 2) = make_float2(s[n][ri * 2], s[n][ri * 2 + 1]);
        fence_reads_before_copies();
        __syncthreads();                                                 // partials written; the stage of `tile` is free
        if (tile >= 0) load(tile + kStages);
        // ---- softmax of tile + 1, a row by TPR neighbouring threads
        const int key = sc * 2, j = k_lo + (tile + 1) * kKeys + key;
        float2 x = *reinterpret_cast<const float2*>(sS + srow * kScorePitch + key);
#pragma unroll
        for (int q = 1; q < 4; ++q) {
            const float2 y = *reinterpret_cast<const float2*>(sS + (q * R + srow) * kScorePitch + key);
            x.x += y.x; x.y += y.y;
        }
        x.x = j >= lo && j < k_hi ? x.x * p.scale_log2 : -CUDART_INF_F;
        x.y = j + 1 >= lo && j + 1 < k_hi ? x.y * p.scale_log2 : -CUDART_INF_F;
        float mx = fmaxf(x.x, x.y);
#pragma unroll
        for (int d = 1; d < TPR; d <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
        float corr = 1.f;
        if (mx > m_run + 8.f) {                                          // (the same for the whole row)
            corr = exp2f(m_run - mx);
            m_run = mx;
        }
        const float base = m_run == -CUDART_INF_F ? 0.f : m_run;
        x.x = exp2f(x.x - base);
        x.y = exp2f(x.y - base);
        l_run = l_run * corr + x.x + x.y;
        *reinterpret_cast<uint32_t*>(sP + srow * kPPitch + key * 2) = pack_bf16x2(x.x, x.y);
        if (sc == 0) sCorr[srow] = corr;
        __syncthreads();
    }
    // ---- denominators
#pragma unroll
    for (int d = 1; d < TPR; d <<= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, d);
    __syncthreads();
    if (sc == 0) {
        sCorr[srow] = l_run;
        sMax[srow] = m_run;
    }
    __syncthreads();
    if (!ok) {                                                           // a copy did not arrive: reported, nothing is stored
        for (int i = 0; i < 200; ++i) __nanosleep(1000);                 // copies still in flight land before the shared memory is reused
        return;
    }
#pragma unroll
    for (int ri = 0; ri < 2; ++ri) {
        const int r = ri * 8 + (lane >> 2), h = h0 + r;
        if (h >= p.Hq) continue;
        const float l = sCorr[r], inv = l > 0.f ? 1.f / l : 0.f;
        float* scr = p.scratch + (((size_t)t * p.Hq + h) * p.nsplit + split) * (a.cpad + 2);
#pragma unroll
        for (int i = 0; i < VT * 2; ++i) {
            const int col = warp * VT * 16 + i * 8 + (lane & 3) * 2;
            if (col < a.cpad) {
                if (p.nsplit > 1)
                    *reinterpret_cast<float2*>(scr + col) = make_float2(o[i][ri * 2], o[i][ri * 2 + 1]);
                else
                    *reinterpret_cast<uint32_t*>(reinterpret_cast<__nv_bfloat16*>(p.out) + (size_t)t * p.ldo + (size_t)h * p.o_head + col) =
                        pack_bf16x2(o[i][ri * 2] * inv, o[i][ri * 2 + 1] * inv);
            }
        }
        if (p.nsplit > 1 && warp == 0 && (lane & 3) == 0) {
            scr[a.cpad] = sMax[r];
            scr[a.cpad + 1] = l;
        }
    }
}

int latent_smem(int k_row) { return kStages * kKeys * k_row * 2 + 4 * kHeads * kScorePitch * 4 + kHeads * kPPitch + 2 * kHeads * 4 + 64 + 128; }

template <int VT, int KQ, bool FULL>
int launch_latent(const LatentKParams& a, cudaStream_t stream) {
    const int smem = latent_smem(a.p.k_row);
    if (smem > 227 * 1024 || a.row / 16 > 4 * KQ) return ERR_UNSUPPORTED;
    auto kern = latent_attention_kernel<VT, KQ, FULL>;
    static std::atomic<uint64_t> configured{0};   // one bit per device; raised to the whole limit once
    int dev = 0;
    OVB_CHECK_CUDA(cudaGetDevice(&dev));
    const uint64_t bit = 1ull << (dev & 63);
    if (!(configured.load(std::memory_order_acquire) & bit)) {
        OVB_CHECK_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
        configured.fetch_or(bit, std::memory_order_release);
    }
    OVB_CHECK_CUDA(launch_pdl(kern, dim3(a.p.T, ceil_div(a.p.Hq, kHeads), a.p.nsplit), dim3(kWarps * 32), (size_t)smem, stream, a));
    return a.p.nsplit > 1 ? launch_decode_combine(a.p, a.cpad, stream) : 0;
}

template <int VT, int KQ>
int launch_latent_sizes(const LatentKParams& a, cudaStream_t stream) {
    return a.row == 64 * KQ && a.cpad == 64 * VT ? launch_latent<VT, KQ, true>(a, stream) : launch_latent<VT, KQ, false>(a, stream);
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
    for (int r = blockIdx.x * 16 + warp; r < min(rows, (int)blockIdx.x * 16 + 16); r += 8) {
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
    if (row % 16 || cpad > 512 || (p.block_size & (p.block_size - 1)) || p.k_row < row || p.k_row % 8 || p.ldq % 8 || p.q_head % 8 || p.ldo % 2 || p.o_head % 2 ||
        (reinterpret_cast<uintptr_t>(p.q) & 15) || (reinterpret_cast<uintptr_t>(p.k_cache) & 15) || (reinterpret_cast<uintptr_t>(p.out) & 3) || p.T > (1 << 30))
        return ERR_UNSUPPORTED;
    LatentKParams a;
    a.p = p;
    a.row = row;
    a.cpad = cpad;
    a.block_shift = 0;
    while ((1 << a.block_shift) < p.block_size) ++a.block_shift;
    a.status = status_word();
    a.p.dv_store = cpad;
    const int keys = p.sliding_window > 0 && p.sliding_window + kKeys - 1 < max_ctx ? p.sliding_window + kKeys - 1 : max_ctx;
    const int tiles = ceil_div(keys, kKeys), ctas = p.T * ceil_div(p.Hq, kHeads);
    const int slots = 148 * 3;   // CTAs that run at a time (registers)
    int best = 1;
    if (max_q_len == 1 && p.T == p.B && p.scratch != nullptr) {
        // shares of the keys: whole waves, a fixed cost of about ten key tiles per CTA and a few more for the merge
        double best_cost = 1e30;
        for (int n = 1; n <= 32 && n <= tiles; ++n) {
            if ((long long)p.T * p.Hq * n * (cpad + 2) * 4 > scratch_bytes) break;
            const double cost = ceil_div(ctas * n, slots) * (ceil_div(tiles, n) + 10.0) + (n > 1 ? 8.0 + 0.5 * n : 0.0);
            if (cost < best_cost) {
                best_cost = cost;
                best = n;
            }
        }
    }
    a.p.nsplit = best;
    a.p.keys_per_split = ceil_div(tiles, best) * kKeys;
    return cpad <= 128 ? launch_latent_sizes<2, 3>(a, stream) : cpad <= 256 ? launch_latent_sizes<4, 5>(a, stream) : launch_latent_sizes<8, 9>(a, stream);
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
    OVB_CHECK_CUDA(launch_pdl(latent_gather_kernel, dim3(ceil_div(rows, 16)), dim3(256), (size_t)(B + 1) * 4, (cudaStream_t)stream, (const uint8_t*)cache,
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
    p.cache_rows = a->cache_rows;
    p.shared = a->cache; p.shared_row = a->row_pitch; p.shared_col = a->key_off; p.q_shared = a->q_rot_off;
    p.block_size = a->block_size; p.sliding_window = a->window; p.causal = 1;
    p.scale_log2 = a->scale * 1.4426950408889634f;
    const int rc = launch_window_tc(p, a->k_head, a->R, a->Dv, (cudaStream_t)stream);
    if (rc == ERR_UNSUPPORTED) set_error("ovb_latent_prefill: sizes %d + %d / %d are not served", a->k_head, a->R, a->Dv);
    return rc;
}

}  // extern "C"
