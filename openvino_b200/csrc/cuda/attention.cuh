// Kernel parameters shared by the attention kernels (attention.cu: mma.sync prefill fallback, split-KV decode;
// attention_sm100.cu: tcgen05 prefill).
#pragma once
#include <cuda_runtime.h>

namespace ovb {

struct PaKParams {
    const void* q;
    void* out;
    const void* k_cache;
    const void* v_cache;
    const int* past_lens;
    const int* subsequence_begins;
    const int* block_indices;
    const int* block_indices_begins;
    float* scratch;
    int B, T, Hq, Hkv;
    int ldq;
    int block_size;
    int sliding_window;
    int nsplit;
    int keys_per_split;
    float scale_log2;
    // dense mode (no paging): k/v are [B, S, H, D] with token pitch ld_kv elements
    int dense_S;
    int ld_kv;
    int causal;
    // u8 KV cache (kv_u8 != 0): k_cache / v_cache hold bytes [block, kv head, slot, D]; k_meta / v_meta hold one fp16 pair
    // (scale, zero point) per (block, kv head, slot): value = (byte - zero point) * scale
    int kv_u8;
    const void* k_meta;
    const void* v_meta;
    // Layout of heads (elements). Query head i of a token starts at column i * q_head, its output row of dv_store columns at
    // column i * o_head of a row of ldo; key / value rows of the paged cache have k_row / v_row elements.
    int q_head, o_head, ldo, dv_store, k_row, v_row;
    // optional output gate: out *= sigmoid(gate[t * ld_gate + head * gate_head + column])
    const void* gate;
    int ld_gate, gate_head;
    int gate_scalar;          // 1: one gate value per head, gate[t * ld_gate + head * gate_head]
    int chunk;                // > 0: a position sees only keys of its own chunk of this many positions (counted from position 0)
    const float* sink;        // [Hq] or NULL: exp(sink[head]) is added to the softmax denominator (no key, no value, not scaled)
    int group;                // query heads per KV head where the kernel takes it at run time
    // Latent attention with expanded heads: keys and values of sequence b, from key kv_first(b) on, are the contiguous rows
    // kv_rows[b] .. of k_cache / v_cache (head h at column h * k_head / h * v_head); a second key part that all heads share is
    // read from the paged cache `shared` (rows of shared_row elements) at column shared_col, and meets the query's columns from q_shared on.
    const int* kv_rows;
    const void* shared;
    int cache_rows;           // rows of the paged caches (0: not known); copies are bounded by it
    int kv_total, kv_ld, k_head, v_head, shared_row, shared_col, q_shared;
};

// First key that position `pos` sees under a sliding window and / or a chunk (0: off); it never decreases with the position.
__host__ __device__ inline int first_visible_key(int pos, int window, int chunk) {
    int lo = window > 0 ? pos - window + 1 : 0;
    if (lo < 0) lo = 0;
    const int start = chunk > 0 ? pos - pos % chunk : 0;
    return lo > start ? lo : start;
}

// First key that is expanded for a sequence: what the window of its first new token reaches, rounded down to whole key tiles.
__host__ __device__ inline int latent_first_key(int past, int window) {
    const int lo = window > 0 ? past - window + 1 : 0;
    return lo > 0 ? lo / 128 * 128 : 0;
}

// tcgen05 / TMA prefill and dense attention (attention_sm100.cu). Returns a negative code when the shape is not one it
// serves (the caller then uses the mma.sync kernel): head size 64 or 128, 16-key pages, 1, 2, 4 or 8 query heads per KV head.
int launch_prefill_tc(const PaKParams& p, int D, int G, bool paged, bool f16, int num_q_tiles, cudaStream_t stream);
// The same kernel with key and value sizes of their own (up to three and two 64-column parts) and any group size up to 16; bf16.
// dk, dv: padded sizes (multiples of 16). dshared > 0: latent attention with expanded heads (PaKParams::kv_rows).
int launch_window_tc(PaKParams p, int dk, int dshared, int dv, cudaStream_t stream);
// Merge of the split-KV partials of a decode batch, scratch [B, Hq, nsplit, dv + 2] (attention.cu).
int launch_decode_combine(const PaKParams& p, int dv, cudaStream_t stream);
// All query heads over one cached row per token whose first dv elements are the value (attention_latent.cu); bf16. cpad: dv padded to 16.
int launch_latent_attention(PaKParams p, int row, int cpad, int max_q_len, int max_ctx, long long scratch_bytes, cudaStream_t stream);
// Split-KV decode with key and value sizes of their own (up to 256) and any group size; bf16, 16-token blocks (attention.cu).
int launch_window_decode(PaKParams p, int dk, int dv, int max_ctx, long long scratch_bytes, cudaStream_t stream);

}  // namespace ovb
