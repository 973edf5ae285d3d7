// The seam between two sublayers of a decoder that normalises before and after each of them, in one kernel:
//
//   x   = sum over the parts of w_j y_j             (one row, or the rows a mixture of experts leaves per token)
//   h  += layernorm(x; post) (+ add)                (residual stream, f32, in place)
//   out = layernorm(h; pre)                         (bf16 or f32, the next sublayer's input)
//
// Layer norm: (x - mean) / sqrt(mean((x - mean)^2) + eps) * w + b, both statistics in f32 from registers (the row is read
// once).  Rows are padded with zeros to a multiple of 8 columns; the statistics run over the first n columns, and the
// padding of w and b is zero, which keeps the padding of h and out zero.  One block per row.
#include "common.cuh"

struct SandwichArgs {
    float* h;                 // [rows, D]
    const void* y;            // [P, D] f32 or bf16, or null: h is only read
    const int* pos;           // [rows * parts] row of y per part (negative: skipped), or null: row * parts + j
    const float* wts;         // [rows * parts] weight per part, or null: 1
    const float* post_w;      // [D] each
    const float* post_b;
    const float* add;         // [D] or null
    const float* pre_w;       // [D] each, or null: no output
    const float* pre_b;
    void* out;                // [rows, D]
    long rows;
    int D, n, parts, y_f32, out_f32;
    float eps;
};

__device__ __forceinline__ float4 ld4(const float* p, int i) { return reinterpret_cast<const float4*>(p)[i]; }

__device__ __forceinline__ float4 ld4_any(const void* p, long row, int D, int i, int f32) {
    if (f32) return reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p) + row * D)[i];
    const uint2 r = reinterpret_cast<const uint2*>(reinterpret_cast<const bf16*>(p) + row * D)[i];
    const float2 a = __bfloat1622float2(*reinterpret_cast<const bf162*>(&r.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const bf162*>(&r.y));
    return make_float4(a.x, a.y, b.x, b.y);
}

// Block-wide sum with one barrier: the caller alternates between two halves of `red` (32 floats each), so a half is written
// again only after a barrier that every thread reaches after reading it.
__device__ __forceinline__ float block_sum_half(float v, float* half) {
    const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, nw = blockDim.x >> 5;
    v = warp_sum(v);
    if (nw == 1) return v;
    if (lane == 0) half[w] = v;
    __syncthreads();
    return warp_sum(lane < nw ? half[lane] : 0.f);
}

// v <- (v - mean) * rstd for the columns below n, 0 beyond
template <int V>
__device__ __forceinline__ void ln_rows(float4 (&v)[V], int n, float eps, float* red) {
    const int nt = blockDim.x;
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < V; ++j) s += v[j].x + v[j].y + v[j].z + v[j].w;      // columns past n hold zeros
    const float mean = block_sum_half(s, red) / (float)n;
    float q = 0.f;
#pragma unroll
    for (int j = 0; j < V; ++j) {
        const int c = (threadIdx.x + j * nt) * 4;
        v[j].x = c + 0 < n ? v[j].x - mean : 0.f;
        v[j].y = c + 1 < n ? v[j].y - mean : 0.f;
        v[j].z = c + 2 < n ? v[j].z - mean : 0.f;
        v[j].w = c + 3 < n ? v[j].w - mean : 0.f;
        q += v[j].x * v[j].x + v[j].y * v[j].y + v[j].z * v[j].z + v[j].w * v[j].w;
    }
    const float rs = 1.f / sqrtf(block_sum_half(q, red + 32) / (float)n + eps);
#pragma unroll
    for (int j = 0; j < V; ++j) { v[j].x *= rs; v[j].y *= rs; v[j].z *= rs; v[j].w *= rs; }
}

template <int V>
__global__ void __launch_bounds__(V == 1 ? 1024 : 512, V == 2 ? 3 : 1) sandwich_norm_kernel(SandwichArgs a) {
    __shared__ float red[64];
    const long row = blockIdx.x;
    const int nvec = a.D >> 2, nt = blockDim.x;
    float4 pw[V], pb[V];                       // the weights do not depend on the previous kernel
    const bool early = V == 1;
    if (early && a.y != nullptr) {
#pragma unroll
        for (int j = 0; j < V; ++j) {
            const int i = threadIdx.x + j * nt;
            if (i < nvec) { pw[j] = ld4(a.post_w, i); pb[j] = ld4(a.post_b, i); }
        }
    }
    pdl_wait();
    pdl_trigger();
    float4 x[V], h[V];
#pragma unroll
    for (int j = 0; j < V; ++j) {
        const int i = threadIdx.x + j * nt;
        x[j] = h[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < nvec) h[j] = reinterpret_cast<const float4*>(a.h + row * a.D)[i];
    }
    if (a.y != nullptr) {
        constexpr int PB = V <= 4 ? 4 : 2;                     // parts in flight together
        for (int p0 = 0; p0 < a.parts; p0 += PB) {
            long src[PB];
            float w[PB];
#pragma unroll
            for (int q = 0; q < PB; ++q) {
                const long k = row * a.parts + p0 + q;
                const bool on = p0 + q < a.parts;
                src[q] = !on ? -1 : a.pos ? (long)a.pos[k] : k;
                w[q] = on && a.wts ? a.wts[k] : 1.f;
            }
#pragma unroll
            for (int j = 0; j < V; ++j) {
                const int i = threadIdx.x + j * nt;
                float4 t[PB];
#pragma unroll
                for (int q = 0; q < PB; ++q)
                    t[q] = i < nvec && src[q] >= 0 ? ld4_any(a.y, src[q], a.D, i, a.y_f32) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                for (int q = 0; q < PB; ++q) {
                    x[j].x += w[q] * t[q].x; x[j].y += w[q] * t[q].y; x[j].z += w[q] * t[q].z; x[j].w += w[q] * t[q].w;
                }
            }
        }
        ln_rows<V>(x, a.n, a.eps, red);
    }
    if (a.y != nullptr || a.add != nullptr) {
#pragma unroll
        for (int j = 0; j < V; ++j) {
            const int i = threadIdx.x + j * nt;
            if (i < nvec) {
                if (a.y != nullptr) {
                    const float4 w = early ? pw[j] : ld4(a.post_w, i), b = early ? pb[j] : ld4(a.post_b, i);
                    h[j].x += x[j].x * w.x + b.x; h[j].y += x[j].y * w.y + b.y;
                    h[j].z += x[j].z * w.z + b.z; h[j].w += x[j].w * w.w + b.w;
                }
                if (a.add != nullptr) {
                    const float4 d = ld4(a.add, i);
                    h[j].x += d.x; h[j].y += d.y; h[j].z += d.z; h[j].w += d.w;
                }
                reinterpret_cast<float4*>(a.h + row * a.D)[i] = h[j];
            }
        }
    }
    if (a.pre_w == nullptr) return;
    ln_rows<V>(h, a.n, a.eps, red);
#pragma unroll
    for (int j = 0; j < V; ++j) {
        const int i = threadIdx.x + j * nt;
        if (i < nvec) {
            const float4 w = ld4(a.pre_w, i), b = ld4(a.pre_b, i);
            const float4 o = make_float4(h[j].x * w.x + b.x, h[j].y * w.y + b.y, h[j].z * w.z + b.z, h[j].w * w.w + b.w);
            if (a.out_f32) {
                reinterpret_cast<float4*>(reinterpret_cast<float*>(a.out) + row * a.D)[i] = o;
            } else {
                uint2 r;
                *reinterpret_cast<bf162*>(&r.x) = __floats2bfloat162_rn(o.x, o.y);
                *reinterpret_cast<bf162*>(&r.y) = __floats2bfloat162_rn(o.z, o.w);
                reinterpret_cast<uint2*>(reinterpret_cast<bf16*>(a.out) + row * a.D)[i] = r;
            }
        }
    }
}

extern "C" int tsb_sandwich_norm(const SandwichArgs* args, void* stream) {
    const SandwichArgs& a = *args;
    TSB_CHECK_ARG(a.D > 0 && a.D % 8 == 0 && a.n > 0 && a.n <= a.D && a.parts > 0, "sandwich_norm: bad shape D=%d n=%d parts=%d", a.D, a.n, a.parts);
    TSB_CHECK_ARG(a.y == nullptr || (a.post_w && a.post_b), "sandwich_norm: the post norm's weights are missing");
    TSB_CHECK_ARG(a.pre_w == nullptr || (a.pre_b && a.out), "sandwich_norm: the pre norm's bias or output is missing");
    if (a.rows == 0) return TSB_OK;
    cudaStream_t s = (cudaStream_t)stream;
    const int nvec = a.D / 4;
    const dim3 grid((unsigned)a.rows);
    // few rows (decode): a float4 per thread, for latency; many rows: two or more each (measured at 8192 x 2048, five parts:
    // one 151 us, two at three CTAs per SM 105 us, three 155, four 150)
    if (nvec <= 256 || (a.rows < 296 && nvec <= 1024)) {
        TSB_CHECK_CUDA(tsb_launch(sandwich_norm_kernel<1>, grid, dim3((nvec + 31) & ~31), 0, s, a));
    } else {
        TSB_CHECK_ARG(nvec <= 4096, "sandwich_norm: rows of %d columns (limit 16384)", a.D);
        const int v = nvec <= 1024 ? 2 : nvec <= 2048 ? 4 : 8;
        const dim3 block((((nvec + v - 1) / v) + 31) & ~31);
        if (v == 2) TSB_CHECK_CUDA(tsb_launch(sandwich_norm_kernel<2>, grid, block, 0, s, a));
        else if (v == 4) TSB_CHECK_CUDA(tsb_launch(sandwich_norm_kernel<4>, grid, block, 0, s, a));
        else TSB_CHECK_CUDA(tsb_launch(sandwich_norm_kernel<8>, grid, block, 0, s, a));
    }
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}
