// Argument block of the attention entry points (shared by the translation units that launch them).
#pragma once
#include "common.cuh"

struct AttnArgs {
    const bf16* q;            // [Tq, Hq, Dh]
    const bf16* k_cache;
    const bf16* v_cache;
    bf16* out;                // [Tq, Hq, Dh]
    const int* block_table;   // [B, max_pages]
    const int* kv_lens;       // [B] tokens in the cache for this sequence (including the new ones)
    const int* cu_q;          // [B + 1] query offsets (prefill); null for decode (one query per sequence)
    const float* sinks;       // [Hq] or null
    float* part_o;            // decode scratch [B, Hq, splits, Dh]
    float* part_ml;           // decode scratch [B, Hq, splits, 2]
    float scale;
    float softcap;            // 0 = off
    int window;               // 0 = full causal
    int B, Hq, Hkv, Dh, page_size, max_pages, splits;
    // Prefill only.  Context parallelism runs the kernel once per KV shard and merges the partial results:
    const int* q_pos0;        // [B] cache position of each sequence's first query, or null = kv_len - q_len
    float* lse_out;           // [Tq, Hq] log-sum-exp of the scaled scores seen by this call (-inf if none), or null
    // Decode only: the output again as int8 groups of 32 with (scale, sum), the form the following
    // quantised projection reads, so that no separate quantise launch is needed.  Null = not wanted.
    int8_t* out_q;            // [B, Hq * Dh]
    float2* out_ds;           // [B, Hq * Dh / 32]
    // Set by the launcher, not the caller: per (sequence, KV head) arrival counters.  When present, the
    // CTA that finishes a head group last merges the split partials itself and no combine kernel runs.
    unsigned* ticket;
    // Decode: positions per split fixed by the caller (a multiple of 32), so that a CTA's range and its block-table
    // entries do not wait for the sequence length; 0 = derive it from the length (ceil(span / splits), rounded to 32).
    int split_len;
    // Output gate: head h of query row t is multiplied by sigmoid(gate[t * gate_tok + h]) (t: packed query row; decode:
    // the sequence).  Null: none.
    const void* gate;
    long gate_tok;            // elements between query rows
    int gate_f32;
    int Dv;                   // value head size (0 = Dh): v_cache [slots, Hkv, Dv], out [Tq, Hq, Dv]
    // Elements between slots where the rows of a slot are not dense (attention_vd.cu and the 32-bit kernel): 0 = Hkv * Dh
    // and Hkv * Dv.  Multiples of 8.
    long k_ld, v_ld;
    // The forms below are served by attention_vd.cu and the 32-bit kernel.
    int keep_first;           // with a window: these first positions stay visible as well
    const float* slopes;      // [Hq] or null: slopes[h] * (query position - key position) is taken off the scaled score
    int gate_cols;            // 1: the gate has a value per output column, gate[t * gate_tok + h * Dv + d]
    int kv_scale;             // != 0: a row of k_cache is key and value at once (Dv = Dh; v_cache is not read), and the score of a
                              // key is multiplied by the f32 number that starts at element kv_scale of its row
    const float* log_r1;      // [Hq] or null: log_r1[h] ln(1 + log_r2[h] (query position - key position)) is taken off the score
    const float* log_r2;
    const float* sig_bias;    // [Hq] or null: no softmax; a visible key's weight is sigmoid(score + sig_bias[h])
};

// Whether only the kernels for head sizes of their own know a form that these arguments ask for.
static inline bool attn_needs_vd(const AttnArgs& a) {
    return (a.Dv != 0 && a.Dv != a.Dh) || a.k_ld != 0 || a.v_ld != 0 || a.keep_first > 0 || a.slopes != nullptr || a.gate_cols || a.kv_scale ||
           a.log_r1 != nullptr || a.sig_bias != nullptr || (a.Dh != 64 && a.Dh != 128 && a.Dh != 256 && a.Dh != 512);
}

#ifdef __CUDACC__
// the gate of head h, or with gate_cols of its column d
__device__ __forceinline__ float attn_gate(const AttnArgs& a, long t, int h, int d = 0) {
    if (a.gate == nullptr) return 1.f;
    const long i = t * a.gate_tok + (a.gate_cols ? (long)h * a.Dv + d : h);
    const float g = a.gate_f32 ? reinterpret_cast<const float*>(a.gate)[i] : bf2f(reinterpret_cast<const bf16*>(a.gate)[i]);
    return 1.f / (1.f + __expf(-g));
}
__device__ __forceinline__ const float* attn_key_factor(const AttnArgs& a, long slot) {
    return reinterpret_cast<const float*>(a.k_cache + slot * a.k_ld + a.kv_scale);
}
#endif

// attention_vd.cu: key and value head sizes of their own (multiples of 16)
int tsb_attn_prefill_vd_launch(const AttnArgs& a, int max_q, cudaStream_t s);
int tsb_attn_decode_vd_launch(const AttnArgs& a, cudaStream_t s);         // the caller launches the combine

// attention_decode_mma.cu: the tensor-core split kernel for decode batches (head sizes 64 / 128, up to 16 query heads
// per KV head); the caller launches the combine unless `*merged` comes back true (splits merged by a thread-block cluster).
bool tsb_attn_decode_mma_supported(const AttnArgs& a);
int tsb_attn_decode_mma_launch(const AttnArgs& a, cudaStream_t s, bool* merged);
int tsb_attn_decode_mma_fp8_launch(const AttnArgs& a, cudaStream_t s);      // e4m3 pages; the caller launches the combine
