// Arguments and element functions of the generalized delta rule's kernels (general_delta.cu, general_delta_chunk.cu).
#pragma once
#include "common.cuh"

struct GdrArgs {
    const void* y; long y_s; int y_f32;      // rows [r | k | v | a' | g | t]: five parts of H * D, then the decay's low rank part
    const float* z; long z_s;                // prompts: the decay's projection [T, H * D] without w0
    const void* w2; int w2_f32;              // short steps: [H * D, rank], z = w2 tanh(t)
    const float* w0; const float* ab; const float* norm_w;      // [H * D]
    float* state; long state_s;              // slot stride
    const int* cu_q; const long* seq_slots;
    float* pack;                             // scan: [T + 1, H, 5, D], u | w | a | r | v * |k|, record T changes nothing; chunks: records
    float* link;                             // [T + 1, H, 4]: u' . (a u) and u' . u with the next token's key u'
    float* core;                             // [T, H, D]
    void* out; long out_s; int out_f32;      // [T, H * D]
    int T, B, H, D, n, rank;
    float eps;
};

constexpr float GDR_KEY_EPS = 1e-6f;

__device__ __forceinline__ float gd_ld(const void* p, long i, int f32) {
    return f32 ? reinterpret_cast<const float*>(p)[i] : bf2f(reinterpret_cast<const bf16*>(p)[i]);
}
__device__ __forceinline__ float4 gd_ld4(const void* p, long i, int f32) {
    if (f32) return *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p) + i);
    const uint2 r = *reinterpret_cast<const uint2*>(reinterpret_cast<const bf16*>(p) + i);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const bf162*>(&r.x)), b = __bfloat1622float2(*reinterpret_cast<const bf162*>(&r.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void gd_st(void* p, long i, int f32, float v) {
    if (f32) reinterpret_cast<float*>(p)[i] = v;
    else reinterpret_cast<bf16*>(p)[i] = f2bf(v);
}
__device__ __forceinline__ float gd_sigmoid(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float gd_decay(float z) {
    constexpr float C = 0.60653065971263342f;            // e^(-1/2)
    return expf(-C * gd_sigmoid(z));
}

static inline int gdr_check(const GdrArgs& a, const char* what) {
    TSB_CHECK_ARG(a.H > 0 && a.D >= 32 && a.D <= 256 && a.D % 32 == 0 && a.n > 0 && a.n <= a.D && a.rank >= 0 && a.rank <= 4096,
                  "%s: heads %d of %d (true size %d), rank %d", what, a.H, a.D, a.n, a.rank);
    TSB_CHECK_ARG(a.B <= 65535 && a.H <= 65535 && a.state_s % 4 == 0, "%s: %d sequences, %d heads", what, a.B, a.H);
    return TSB_OK;
}

// general_delta.cu: norm and gate of the recurrence's results
int tsb_gdr_finish_launch(const GdrArgs& a, cudaStream_t s);
