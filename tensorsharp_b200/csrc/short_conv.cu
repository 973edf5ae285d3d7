// Causal convolution over time on every channel of a projection, without an activation, in one kernel with its state:
//
//   o_t = bias + sum_j w[j] u_(t - K + 1 + j)                  (zeros ahead of a sequence's start)
//
// `state` holds the last K - 1 inputs of each slot's sequence (f32, [K - 1][C], oldest first).  A thread has four channels and up to
// `span` >= K - 1 consecutive tokens of one sequence; the first run of a sequence is the only one that reads the slot's old values,
// and it writes the new ones.
//
// Results go to rows [T, C]; to blocks of columns one below the other, row (c / block) * T + t (what a product with a matrix per
// block reads); or, for attention, queries to rows [T, nq] times the position's temperature 1 + coef ln(floor((p + 1) / every) + 1),
// keys and values to their slots of the paged caches.
#include "common.cuh"

struct ShortConvArgs {
    const void* x; long x_s; int x_f32;
    const float* w;            // [K][C]
    const float* bias;         // [C] or null
    float* state; long state_s;
    const int* cu_q; const long* seq_slots;
    void* out; long out_s; int out_f32;
    int block;                 // 0, or the size of a block of columns
    // attention: channels [q (nq) | k (nk) | v]
    const int* pos; const long* slot;
    void* k_cache; void* v_cache;        // null: queries only
    int nq, nk;
    float qt_coef, qt_every;   // qt_every 0: no temperature
    int T, C, K, B, span;
};

namespace {
// four values as they are stored
template <bool F32> struct Raw4 {
    uint2 r;
    __device__ __forceinline__ void load(const void* p, long at) { r = *reinterpret_cast<const uint2*>(reinterpret_cast<const bf16*>(p) + at); }
    __device__ __forceinline__ float4 get() const {
        const float2 a = __bfloat1622float2(*reinterpret_cast<const bf162*>(&r.x)), b = __bfloat1622float2(*reinterpret_cast<const bf162*>(&r.y));
        return make_float4(a.x, a.y, b.x, b.y);
    }
};
template <> struct Raw4<true> {
    float4 r;
    __device__ __forceinline__ void load(const void* p, long at) { r = *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p) + at); }
    __device__ __forceinline__ float4 get() const { return r; }
};
template <bool F32>
__device__ __forceinline__ float4 sc_ld4(const void* p, long at) {
    Raw4<F32> x;
    x.load(p, at);
    return x.get();
}
__device__ __forceinline__ void sc_st4(void* p, long at, int f32, float4 o) {
    if (f32) {
        *reinterpret_cast<float4*>(reinterpret_cast<float*>(p) + at) = o;
    } else {
        uint2 r;
        *reinterpret_cast<bf162*>(&r.x) = __floats2bfloat162_rn(o.x, o.y);
        *reinterpret_cast<bf162*>(&r.y) = __floats2bfloat162_rn(o.z, o.w);
        *reinterpret_cast<uint2*>(reinterpret_cast<bf16*>(p) + at) = r;
    }
}
__device__ __forceinline__ void sc_fma(float4& x, float4 w, float4 t) {
    x.x = fmaf(w.x, t.x, x.x); x.y = fmaf(w.y, t.y, x.y); x.z = fmaf(w.z, t.z, x.z); x.w = fmaf(w.w, t.w, x.w);
}
}  // namespace

// Grid (runs, pieces of 512 channels), 128 threads.
template <int H, bool QKV, bool F32>
__global__ void __launch_bounds__(128) short_conv_kernel(ShortConvArgs a) {
    const int c = (blockIdx.y * 128 + threadIdx.x) * 4;
    int b = 0;
    long r0 = 0;
    if (a.T == a.B) {
        b = blockIdx.x;
        r0 = b;
    } else {
        long before = 0;
        for (;; ++b) {
            if (b == a.B) return;
            const long n = a.cu_q[b + 1] - a.cu_q[b], runs = (n + a.span - 1) / a.span;
            if ((long)blockIdx.x < before + runs) break;
            before += runs;
        }
        r0 = a.cu_q[b] + ((long)blockIdx.x - before) * a.span;
    }
    if (c >= a.C) return;
    const long first = a.cu_q[b], end = a.cu_q[b + 1], r1 = min(end, r0 + a.span);
    float* st = a.state + a.seq_slots[b] * a.state_s + c;
    float4 w[H + 1], hist[H > 0 ? H : 1], bias = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int k = 0; k <= H; ++k) w[k] = *reinterpret_cast<const float4*>(a.w + (long)k * a.C + c);
    if (a.bias != nullptr) bias = *reinterpret_cast<const float4*>(a.bias + c);
    if (r0 == first) {
#pragma unroll
        for (int k = 0; k < H; ++k) hist[k] = *reinterpret_cast<const float4*>(st + (long)k * a.C);
    }
    // where the results go: base, elements per token or per slot
    void* dst = a.out;
    long at = c, step = a.out_s;
    const long* index = nullptr;
    float coef = 0.f;
    if (QKV) {
        if (c < a.nq) {
            coef = a.qt_every > 0.f ? a.qt_coef : 0.f;
        } else if (c < a.nq + a.nk) {
            dst = a.k_cache; at = c - a.nq; step = a.nk; index = a.slot;
        } else {
            dst = a.v_cache; at = c - a.nq - a.nk; step = a.C - a.nq - a.nk; index = a.slot;
        }
    } else if (a.block > 0) {
        at = (long)(c / a.block) * a.T * a.block + c % a.block;
        step = a.block;
    }
    pdl_wait();
    pdl_trigger();
    if (r0 != first) {
#pragma unroll
        for (int k = 0; k < H; ++k) hist[k] = sc_ld4<F32>(a.x, (r0 - H + k) * a.x_s + c);
    }
    constexpr int U = F32 ? 4 : 8;                             // rows loaded together
    for (long row = r0; row < r1; row += U) {
        Raw4<F32> x[U];
        int at_pos[U];                                         // slot or position, whichever these channels need
#pragma unroll
        for (int q = 0; q < U; ++q) {
            const long t = min(row + q, r1 - 1);
            x[q].load(a.x, t * a.x_s + c);
            if (QKV) at_pos[q] = index != nullptr ? (int)index[t] : coef != 0.f ? a.pos[t] : 0;
        }
#pragma unroll
        for (int q = 0; q < U; ++q) {
            if (row + q >= r1) break;
            const float4 u = x[q].get();
            float4 o = bias;
#pragma unroll
            for (int k = 0; k < H; ++k) sc_fma(o, w[k], hist[k]);
            sc_fma(o, w[H], u);
#pragma unroll
            for (int k = 0; k + 1 < H; ++k) hist[k] = hist[k + 1];
            if (H > 0) hist[H - 1] = u;
            if (QKV && coef != 0.f) {
                const float m = 1.f + coef * logf(floorf(((float)at_pos[q] + 1.f) / a.qt_every) + 1.f);
                o = make_float4(o.x * m, o.y * m, o.z * m, o.w * m);
            }
            sc_st4(dst, at + (QKV && index != nullptr ? (long)at_pos[q] : row + q) * step, a.out_f32, o);
        }
    }
    if (H == 0 || r0 != first) return;
    if (r1 < end) {
#pragma unroll
        for (int k = 0; k < H; ++k) *reinterpret_cast<float4*>(st + (long)k * a.C) = sc_ld4<F32>(a.x, (end - H + k) * a.x_s + c);
    } else {
#pragma unroll
        for (int k = 0; k < H; ++k) *reinterpret_cast<float4*>(st + (long)k * a.C) = hist[k];
    }
}

extern "C" int tsb_short_conv(const ShortConvArgs* args, void* stream) {
    ShortConvArgs a = *args;
    TSB_CHECK_ARG(a.K >= 1 && a.K <= 8, "short_conv: %d taps (1 to 8)", a.K);
    TSB_CHECK_ARG(a.C > 0 && a.C % 4 == 0 && a.x_s % 4 == 0 && a.state_s % 4 == 0 && a.out_s % 4 == 0 && a.block % 4 == 0 && (a.block == 0 || a.C % a.block == 0),
                  "short_conv: %d channels in blocks of %d", a.C, a.block);
    TSB_CHECK_ARG(a.K == 1 || a.state, "short_conv: no state");
    const bool qkv = a.nq > 0;
    TSB_CHECK_ARG(!qkv || (a.nq % 4 == 0 && a.nk % 4 == 0 && a.pos && a.slot && a.block == 0 && a.nq + a.nk <= a.C && (a.nq == a.C || (a.k_cache && a.v_cache))),
                  "short_conv: %d query and %d key channels of %d", a.nq, a.nk, a.C);
    if (a.T == 0 || a.B == 0) return TSB_OK;
    unsigned runs = (unsigned)a.B;
    a.span = 1;
    if (a.T > a.B) {
        const long per = (long)a.T * (a.C / 4) / (148 * 1024);         // enough threads first, then longer runs
        a.span = per < 4 ? 4 : per > 32 ? 32 : per < 8 ? (int)per : (int)per & ~7;
        if (a.span < a.K - 1) a.span = a.K - 1;
        runs = (unsigned)(a.T / a.span + a.B);
    }
    const dim3 grid(runs, (a.C / 4 + 127) / 128), block(128);
    cudaStream_t s = (cudaStream_t)stream;
    switch (a.K - 1) {
#define GO(H, Q) (a.x_f32 ? tsb_launch(short_conv_kernel<H, Q, true>, grid, block, 0, s, a) : tsb_launch(short_conv_kernel<H, Q, false>, grid, block, 0, s, a))
#define X(H)                                             \
    case H:                                              \
        if (qkv) TSB_CHECK_CUDA(GO(H, true));            \
        else TSB_CHECK_CUDA(GO(H, false));               \
        break;
        X(0) X(1) X(2) X(3) X(4) X(5) X(6) X(7)
#undef X
#undef GO
    }
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}
