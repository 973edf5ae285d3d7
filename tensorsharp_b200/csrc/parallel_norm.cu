// The seam between two layers of a decoder whose sublayers run side by side on one residual stream, in one kernel:
//
//   x     = h + s1 * y1 + s2 * y2                   (residual stream, f32; s: scale per channel; y: the sublayers' outputs)
//   out1  = rmsnorm(x) * w1, then moved towards the previous token's value per channel: v + (v' - v) * shift
//   out2  = rmsnorm(x) * w2
//
// An output without a weight is x itself in the output's type.  The previous token of a sequence's first row in the batch
// comes from `state` (f32, one row per slot), which then receives the unshifted row of the sequence's last token.  The
// new residual goes to a buffer of its own (h_out), so a block may recompute the row ahead of its first one; a block takes
// `span` consecutive rows and hands the normalised row on in registers.
// Rows are padded with zeros to a multiple of 8 columns; the mean of squares runs over the first n.
#include "common.cuh"

struct ParallelNormArgs {
    const float* h;           // [rows, D]
    float* h_out;             // [rows, D] or null (then y1 is null too)
    const void* y1;           // [rows, D] f32 or bf16, or null
    const void* y2;           // the same type, or null
    const float* s1;          // [D] each
    const float* s2;
    const float* w1;          // [D] or null: x itself
    const float* w2;
    void* out1;               // row stride ld1, or null
    void* out2;
    const float* shift;       // [D] or null
    float* state;             // [slots] rows of stride state_s
    const int* cu_q;          // [B + 1]
    const long* seq_slots;    // [B]
    long rows, ld1, ld2, state_s;
    int D, n, B, y_f32, out1_f32, out2_f32, span;
    float eps;
};

namespace {
__device__ __forceinline__ float4 pn_ld4(const float* p, int i) { return reinterpret_cast<const float4*>(p)[i]; }

__device__ __forceinline__ float4 pn_ld4_any(const void* p, long row, int D, int i, int f32) {
    if (f32) return reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p) + row * D)[i];
    const uint2 r = reinterpret_cast<const uint2*>(reinterpret_cast<const bf16*>(p) + row * D)[i];
    const float2 a = __bfloat1622float2(*reinterpret_cast<const bf162*>(&r.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const bf162*>(&r.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void pn_st4(void* p, long at, int i, int f32, float4 o) {
    if (f32) {
        reinterpret_cast<float4*>(reinterpret_cast<float*>(p) + at)[i] = o;
    } else {
        uint2 r;
        *reinterpret_cast<bf162*>(&r.x) = __floats2bfloat162_rn(o.x, o.y);
        *reinterpret_cast<bf162*>(&r.y) = __floats2bfloat162_rn(o.z, o.w);
        reinterpret_cast<uint2*>(reinterpret_cast<bf16*>(p) + at)[i] = r;
    }
}
__device__ __forceinline__ void pn_axpy(float4& x, float4 s, float4 y) {
    x.x = fmaf(s.x, y.x, x.x); x.y = fmaf(s.y, y.y, x.y); x.z = fmaf(s.z, y.z, x.z); x.w = fmaf(s.w, y.w, x.w);
}
__device__ __forceinline__ float4 pn_mul(float4 a, float r, float4 w) { return make_float4(a.x * r * w.x, a.y * r * w.y, a.z * r * w.z, a.w * r * w.w); }

// The new residual row in registers and the reciprocal of its root mean square.  `red`: 64 floats; two calls in a row use
// its halves in turn (`flip`), so one barrier per call is enough.
// The vectors that do not depend on earlier kernels.  With one float4 per thread (decode, narrow rows) they are loaded ahead
// of the dependency wait; otherwise where they are used, for the registers' sake.
template <int V>
struct PnVecs {
    float4 s1, s2, w1, w2, sh;
    __device__ __forceinline__ void load(const ParallelNormArgs& a) {
        const int i = threadIdx.x;
        if (V > 1 || i >= (a.D >> 2)) return;
        if (a.y1 != nullptr) s1 = pn_ld4(a.s1, i);
        if (a.y2 != nullptr) s2 = pn_ld4(a.s2, i);
        if (a.w1 != nullptr) w1 = pn_ld4(a.w1, i);
        if (a.w2 != nullptr) w2 = pn_ld4(a.w2, i);
        if (a.shift != nullptr) sh = pn_ld4(a.shift, i);
    }
    static __device__ __forceinline__ float4 get(const float4& held, const float* p, int i) { return V == 1 ? held : pn_ld4(p, i); }
};

template <int V>
__device__ __forceinline__ float pn_row(const ParallelNormArgs& a, const PnVecs<V>& c, long row, float4 (&x)[V], float* red, int& flip) {
    const int nvec = a.D >> 2, nt = blockDim.x;
    float q = 0.f;
#pragma unroll
    for (int j = 0; j < V; ++j) {
        const int i = threadIdx.x + j * nt;
        x[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < nvec) {
            x[j] = reinterpret_cast<const float4*>(a.h + row * a.D)[i];
            if (a.y1 != nullptr) pn_axpy(x[j], c.get(c.s1, a.s1, i), pn_ld4_any(a.y1, row, a.D, i, a.y_f32));
            if (a.y2 != nullptr) pn_axpy(x[j], c.get(c.s2, a.s2, i), pn_ld4_any(a.y2, row, a.D, i, a.y_f32));
        }
        q += x[j].x * x[j].x + x[j].y * x[j].y + x[j].z * x[j].z + x[j].w * x[j].w;       // padding is zero
    }
    const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, nw = blockDim.x >> 5;
    q = warp_sum(q);
    if (nw > 1) {
        float* half = red + 32 * flip;
        flip ^= 1;
        if (lane == 0) half[w] = q;
        __syncthreads();
        q = warp_sum(lane < nw ? half[lane] : 0.f);
    }
    return 1.f / sqrtf(q / (float)a.n + a.eps);
}
}  // namespace

template <int V>
__global__ void __launch_bounds__(V == 1 ? 1024 : 512) parallel_norm_kernel(ParallelNormArgs a) {
    __shared__ float red[64];
    PnVecs<V> vec;
    vec.load(a);
    pdl_wait();
    pdl_trigger();
    const int nvec = a.D >> 2, nt = blockDim.x;
    const long r0 = (long)blockIdx.x * a.span, r1 = min(a.rows, r0 + a.span);
    int flip = 0, b = 0;
    long first = 0, last = 0;                              // the current sequence's rows
    float4 x[V], prev[V];
    if (a.shift != nullptr) {
        int lo = 0, hi = a.B - 1;                          // the last sequence that starts at or before r0
        while (lo < hi) {
            const int mid = (lo + hi + 1) >> 1;
            if (a.cu_q[mid] <= r0) lo = mid; else hi = mid - 1;
        }
        b = lo;
        first = a.cu_q[b];
        last = a.cu_q[b + 1] - 1;
        if (r0 > first) {                                  // the row ahead of this block's first one
            const float rs = pn_row<V>(a, vec, r0 - 1, x, red, flip);
#pragma unroll
            for (int j = 0; j < V; ++j) {
                const int i = threadIdx.x + j * nt;
                if (i < nvec) prev[j] = pn_mul(x[j], rs, vec.get(vec.w1, a.w1, i));
            }
        }
    }
    for (long row = r0; row < r1; ++row) {
        if (a.shift != nullptr) {
            while (row > last) {
                ++b;
                first = last + 1;
                last = a.cu_q[b + 1] - 1;
            }
            if (row == first) {
                float* st = a.state + a.seq_slots[b] * a.state_s;
#pragma unroll
                for (int j = 0; j < V; ++j) {
                    const int i = threadIdx.x + j * nt;
                    if (i < nvec) prev[j] = reinterpret_cast<const float4*>(st)[i];
                }
                if (last > first) {                        // the slot's next value, by the block that has read the old one
                    const float rs = pn_row<V>(a, vec, last, x, red, flip);
#pragma unroll
                    for (int j = 0; j < V; ++j) {
                        const int i = threadIdx.x + j * nt;
                        if (i < nvec) reinterpret_cast<float4*>(st)[i] = pn_mul(x[j], rs, vec.get(vec.w1, a.w1, i));
                    }
                }
            }
        }
        const float rs = pn_row<V>(a, vec, row, x, red, flip);
#pragma unroll
        for (int j = 0; j < V; ++j) {
            const int i = threadIdx.x + j * nt;
            if (i >= nvec) continue;
            if (a.h_out != nullptr) reinterpret_cast<float4*>(a.h_out + row * a.D)[i] = x[j];
            if (a.out2 != nullptr) pn_st4(a.out2, row * a.ld2, i, a.out2_f32, a.w2 != nullptr ? pn_mul(x[j], rs, vec.get(vec.w2, a.w2, i)) : x[j]);
            if (a.out1 == nullptr) continue;
            float4 v = a.w1 != nullptr ? pn_mul(x[j], rs, vec.get(vec.w1, a.w1, i)) : x[j];
            if (a.shift != nullptr) {
                const float4 m = vec.get(vec.sh, a.shift, i), p = prev[j];
                if (first == last) reinterpret_cast<float4*>(a.state + a.seq_slots[b] * a.state_s)[i] = v;
                prev[j] = v;
                v = make_float4(v.x + (p.x - v.x) * m.x, v.y + (p.y - v.y) * m.y, v.z + (p.z - v.z) * m.z, v.w + (p.w - v.w) * m.w);
            }
            pn_st4(a.out1, row * a.ld1, i, a.out1_f32, v);
        }
    }
}

extern "C" int tsb_parallel_norm(const ParallelNormArgs* args, void* stream) {
    ParallelNormArgs a = *args;
    TSB_CHECK_ARG(a.D > 0 && a.D % 8 == 0 && a.n > 0 && a.n <= a.D && a.ld1 % 4 == 0 && a.ld2 % 4 == 0 && a.state_s % 4 == 0,
                  "parallel_norm: bad shape D=%d n=%d", a.D, a.n);
    TSB_CHECK_ARG(a.y1 == nullptr || (a.s1 && a.h_out), "parallel_norm: the first output's scale or the new residual is missing");
    TSB_CHECK_ARG(a.y2 == nullptr || (a.s2 && a.y1), "parallel_norm: the second output's scale or the first output is missing");
    TSB_CHECK_ARG(a.h_out == nullptr || a.h_out != a.h, "parallel_norm: the residual is not updated in place");
    TSB_CHECK_ARG(a.shift == nullptr || (a.w1 && a.out1 && a.state && a.cu_q && a.seq_slots && a.B > 0), "parallel_norm: the token shift has no state");
    if (a.rows == 0) return TSB_OK;
    cudaStream_t s = (cudaStream_t)stream;
    const int nvec = a.D / 4;
    // few rows: one each, for latency; many rows and a token shift: up to eight in a row per block, since each block
    // computes one row twice
    a.span = 1;
    if (a.shift != nullptr && a.rows > a.B) {
        const long per = a.rows / 592;
        a.span = per < 1 ? 1 : per > 8 ? 8 : (int)per;
    }
    const dim3 grid((unsigned)((a.rows + a.span - 1) / a.span));
    if (nvec <= 256 || (a.rows < 296 && nvec <= 1024)) {
        TSB_CHECK_CUDA(tsb_launch(parallel_norm_kernel<1>, grid, dim3((nvec + 31) & ~31), 0, s, a));
    } else {
        TSB_CHECK_ARG(nvec <= 4096, "parallel_norm: rows of %d columns (limit 16384)", a.D);
        const int v = nvec <= 1024 ? 2 : nvec <= 2048 ? 4 : 8;
        const dim3 block((((nvec + v - 1) / v) + 31) & ~31);
        if (v == 2) TSB_CHECK_CUDA(tsb_launch(parallel_norm_kernel<2>, grid, block, 0, s, a));
        else if (v == 4) TSB_CHECK_CUDA(tsb_launch(parallel_norm_kernel<4>, grid, block, 0, s, a));
        else TSB_CHECK_CUDA(tsb_launch(parallel_norm_kernel<8>, grid, block, 0, s, a));
    }
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}
