// Paged attention for any head sizes, in fp32 arithmetic throughout, over fp32 or bf16 storage: the kernel of the 32-bit mode and
// of the shapes that the tensor-core kernels (attention.cu, attention_sm100.cu, attention_latent.cu) do not serve.
//
// One CTA per (token, query head). Keys are taken 128 at a time: one thread per key for the scores, running maximum and sum over
// the CTA, then one thread per value column. Value rows may lie inside the key rows (latent attention caches one row per token
// and uses its first part as the value).
#include <math_constants.h>

#include "attention.cuh"
#include "debug_bounds.cuh"
#include "sm100_ptx.cuh"
#include "store_types.cuh"

namespace ovb {

OVB_DEBUG_LIMITS_DEFINE

namespace {

constexpr int kThreads = 128;
constexpr int kMaxV = 8;      // value columns per thread

template <class E>
__global__ void __launch_bounds__(kThreads) attention_exact_kernel(ovb_wattn_args p) {
    pdl_enter_attn();
    extern __shared__ float sq[];            // [Dk]
    __shared__ float sp[kThreads], red[kThreads / 32];
    __shared__ int s_b;
    const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    find_sequence(p.subsequence_begins, p.B, t, &s_b);
    const E* q = reinterpret_cast<const E*>(p.q) + (size_t)t * p.ldq + (size_t)h * p.q_head;
    for (int i = tid; i < p.Dk; i += kThreads) sq[i] = ld_f32(q + i) * p.scale;
    __syncthreads();
    const int b = s_b, kvh = h / (p.Hq / p.Hkv);
    const int pos = p.past_lens[b] + t - p.subsequence_begins[b];
    const int* blocks = p.block_indices + p.block_indices_begins[b];
    const int lo = first_visible_key(pos, p.window, p.chunk);
    auto row_of = [&](int j) {
        const int blk = OVB_DBG_BLOCK(blocks[j / p.block_size]);
        return ((size_t)blk * p.Hkv + kvh) * p.block_size + j % p.block_size;
    };
    auto reduce = [&](float v, bool is_max) {
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float w = __shfl_xor_sync(0xffffffffu, v, o);
            v = is_max ? fmaxf(v, w) : v + w;
        }
        __syncthreads();
        if ((tid & 31) == 0) red[tid >> 5] = v;
        __syncthreads();
        v = red[0];
#pragma unroll
        for (int i = 1; i < kThreads / 32; ++i) v = is_max ? fmaxf(v, red[i]) : v + red[i];
        return v;
    };
    float acc[kMaxV] = {}, m = -CUDART_INF_F, l = 0.f;
    for (int j0 = lo; j0 <= pos; j0 += kThreads) {
        const int j = j0 + tid;
        float s = -CUDART_INF_F;
        if (j <= pos) {
            const E* k = reinterpret_cast<const E*>(p.k) + row_of(j) * p.k_row;
            s = 0.f;
            for (int i = 0; i < p.Dk; i += 4) {
                const float4 kv = ld4_f32(k + i);
                s = fmaf(sq[i], kv.x, fmaf(sq[i + 1], kv.y, fmaf(sq[i + 2], kv.z, fmaf(sq[i + 3], kv.w, s))));
            }
        }
        const float m_new = fmaxf(m, reduce(s, true));      // at least one key of the tile is visible
        const float e = j <= pos ? expf(s - m_new) : 0.f;
        const float corr = m == -CUDART_INF_F ? 0.f : expf(m - m_new);
        l = l * corr + reduce(e, false);
        m = m_new;
        sp[tid] = e;
        __syncthreads();
        const int n = min(kThreads, pos - j0 + 1);
#pragma unroll
        for (int i = 0; i < kMaxV; ++i) acc[i] *= corr;
        for (int jj = 0; jj < n; ++jj) {
            const E* v = reinterpret_cast<const E*>(p.v) + row_of(j0 + jj) * p.v_row;
#pragma unroll
            for (int i = 0; i < kMaxV; ++i)
                if (tid + i * kThreads < p.Dv) acc[i] = fmaf(sp[jj], ld_f32(v + tid + i * kThreads), acc[i]);
        }
        __syncthreads();
    }
    if (p.sink) l += expf(p.sink[h] - m);
    E* out = reinterpret_cast<E*>(p.out) + (size_t)t * p.ldo + (size_t)h * p.o_head;
    const E* gate = p.gate ? reinterpret_cast<const E*>(p.gate) + (size_t)t * p.ld_gate + (size_t)h * p.gate_head : nullptr;
#pragma unroll
    for (int i = 0; i < kMaxV; ++i) {
        const int d = tid + i * kThreads;
        if (d < p.Dv) {
            float o = acc[i] / l;
            if (gate) o *= 1.f / (1.f + expf(-ld_f32(gate + (p.gate_scalar ? 0 : d))));
            st_f32(out + d, o);
        }
    }
}

}  // namespace

int launch_attention_exact(const ovb_wattn_args& a, cudaStream_t stream) {
    OVB_REQUIRE(a.Dk % 4 == 0 && a.k_row % 4 == 0 && a.Dk <= 8192, "ovb_window_attention: key rows must be padded to a multiple of 4 elements");
    if (a.Dv > kMaxV * kThreads) {
        set_error("ovb_window_attention: value size %d above %d", a.Dv, kMaxV * kThreads);
        return ERR_UNSUPPORTED;
    }
    return dispatch_store(a.dtype, "ovb_window_attention", [&](auto e) -> int {
        using E = decltype(e);
        OVB_CHECK_CUDA(launch_pdl(attention_exact_kernel<E>, dim3(a.T, a.Hq), dim3(kThreads), (size_t)a.Dk * 4, stream, a));
        return 0;
    });
}

}  // namespace ovb

#ifdef OVB_DEBUG_BOUNDS
extern "C" int ovb_debug_set_limits_exact(const ovb::DebugLimits* l) {
    OVB_CHECK_CUDA(cudaMemcpyToSymbol(ovb::g_dbg_limits, l, sizeof(*l)));
    return 0;
}
#endif

extern "C" int ovb_window_attention(const ovb_wattn_args* a, ovb_stream_t stream) {
    using namespace ovb;
    OVB_REQUIRE(a && a->q && a->out && a->k && a->v, "ovb_window_attention: null operand");
    OVB_REQUIRE(a->past_lens && a->subsequence_begins && a->block_indices && a->block_indices_begins, "ovb_window_attention: null batch descriptor");
    OVB_REQUIRE(a->B > 0 && a->T > 0 && a->Hkv > 0 && a->Hq > 0 && a->Hq % a->Hkv == 0 && a->Dk > 0 && a->Dv > 0 && a->block_size > 0,
                "ovb_window_attention: bad sizes");
    if (a->dtype == OVB_DT_BF16 && !a->exact) {      // the tensor-core kernels, where they serve the sizes
        PaKParams p;
        memset(&p, 0, sizeof(p));
        p.q = a->q; p.out = a->out; p.k_cache = a->k; p.v_cache = a->v; p.gate = a->gate;
        p.past_lens = a->past_lens; p.subsequence_begins = a->subsequence_begins;
        p.block_indices = a->block_indices; p.block_indices_begins = a->block_indices_begins;
        p.scratch = a->scratch;
        p.cache_rows = a->cache_rows;
        p.B = a->B; p.T = a->T; p.Hq = a->Hq; p.Hkv = a->Hkv; p.group = a->Hq / a->Hkv;
        p.ldq = a->ldq; p.q_head = a->q_head; p.ldo = a->ldo; p.o_head = a->o_head; p.k_row = a->k_row; p.v_row = a->v_row;
        p.ld_gate = a->ld_gate; p.gate_head = a->gate_head; p.gate_scalar = a->gate_scalar;
        p.block_size = a->block_size; p.sliding_window = a->window; p.chunk = a->chunk; p.sink = a->sink; p.causal = 1;
        p.scale_log2 = a->scale * 1.4426950408889634f;
        const bool decode = a->max_q_len == 1 && a->T == a->B;
        const int rc = a->k == a->v ? (a->Hkv == 1 && a->gate == nullptr && a->chunk == 0 && a->sink == nullptr ? launch_latent_attention(p, a->Dk, (a->Dv + 15) / 16 * 16, a->max_q_len, a->max_context_len,
                                                                                                   a->scratch_bytes, (cudaStream_t)stream) : ERR_UNSUPPORTED)
                     : decode ? launch_window_decode(p, a->Dk, a->Dv, a->max_context_len, a->scratch_bytes, (cudaStream_t)stream)
                              : a->scale > 0.f ? launch_window_tc(p, a->Dk, 0, (a->Dv + 15) / 16 * 16, (cudaStream_t)stream) : ERR_UNSUPPORTED;
        if (rc != ERR_UNSUPPORTED) return rc;
    }
    return launch_attention_exact(*a, (cudaStream_t)stream);
}
