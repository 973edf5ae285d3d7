// The seam of a decoder that normalises its sublayers' outputs (and only those), in one kernel:
//
//   x   = sum over the parts of w_j y_j             (one row, or the rows a mixture of experts leaves per token; a part with a
//                                                    negative id is the sublayer's input itself: an identity expert)
//   x   = mix (rms(x) b1 + rms(z) b2)               (two branches side by side, each with a norm of its own; optional)
//   h  += rms(x) post                               (residual stream, f32, in place)
//   out = h, or rms(h) pre                          (bf16 or f32: the next sublayer reads the stream itself)
//
// rms(x) = x / sqrt(mean(x^2) + eps), statistics in f32 from registers; every row is read once.  Rows are padded with zeros
// to a multiple of 8 columns, the means run over the first n.  One block per row.
#include "common.cuh"

struct PostNormArgs {
    float* h;                 // [rows, D]
    const void* y;            // [P, D] f32 or bf16, or null: h is only read
    const void* z;            // [rows, D] of the same type, or null: one branch
    const int* ids;           // [rows * parts] or null: no identity parts
    const int* pos;           // [rows * parts] row of y per part, or null: row * parts + j
    const float* wts;         // [rows * parts] weight per part, or null: 1
    const float* b1;          // [D] each
    const float* b2;
    const float* post;
    const float* pre;         // or null: out = h
    void* out;                // [rows, D] or null
    long rows;
    int D, n, parts, y_f32, out_f32;
    float eps, mix;
};

namespace {
__device__ __forceinline__ float4 po_ld4(const float* p, int i) { return reinterpret_cast<const float4*>(p)[i]; }
__device__ __forceinline__ float4 po_ld4_any(const void* p, long row, int D, int i, int f32) {
    if (f32) return reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p) + row * D)[i];
    const uint2 r = reinterpret_cast<const uint2*>(reinterpret_cast<const bf16*>(p) + row * D)[i];
    const float2 a = __bfloat1622float2(*reinterpret_cast<const bf162*>(&r.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const bf162*>(&r.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ float po_sq(float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
__device__ __forceinline__ void po_axpy(float4& x, float w, float4 t) {
    x.x = fmaf(w, t.x, x.x); x.y = fmaf(w, t.y, x.y); x.z = fmaf(w, t.z, x.z); x.w = fmaf(w, t.w, x.w);
}

// Block-wide sums of two values with one barrier; consecutive calls use different thirds of `red` (64 floats each).
__device__ __forceinline__ float2 po_sum2(float2 v, float* part) {
    const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, nw = blockDim.x >> 5;
    v.x = warp_sum(v.x);
    v.y = warp_sum(v.y);
    if (nw == 1) return v;
    if (lane == 0) { part[w] = v.x; part[32 + w] = v.y; }
    __syncthreads();
    return make_float2(warp_sum(lane < nw ? part[lane] : 0.f), warp_sum(lane < nw ? part[32 + lane] : 0.f));
}
}  // namespace

// V float4s per thread.  With one each (decode, narrow rows) the weight vectors are loaded ahead of the dependency wait.
template <int V>
__global__ void __launch_bounds__(V == 1 ? 1024 : 512, V == 2 ? 2 : 1) post_norm_kernel(PostNormArgs a) {
    __shared__ float red[192];
    const long row = blockIdx.x;
    const int nvec = a.D >> 2, nt = blockDim.x;
    const float inv_n = 1.f / (float)a.n;
    float4 w1, w2, wp, wo;
    w1 = w2 = wp = wo = make_float4(0.f, 0.f, 0.f, 0.f);
    if (V == 1 && (int)threadIdx.x < nvec) {
        if (a.z != nullptr) { w1 = po_ld4(a.b1, threadIdx.x); w2 = po_ld4(a.b2, threadIdx.x); }
        if (a.y != nullptr) wp = po_ld4(a.post, threadIdx.x);
        if (a.pre != nullptr) wo = po_ld4(a.pre, threadIdx.x);
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
        float2 ss = make_float2(0.f, 0.f);
        if (a.z != nullptr) {
            float4 z[V];
#pragma unroll
            for (int j = 0; j < V; ++j) {
                const int i = threadIdx.x + j * nt;
                z[j] = make_float4(0.f, 0.f, 0.f, 0.f);
                if (i < nvec) {
                    x[j] = po_ld4_any(a.y, row, a.D, i, a.y_f32);
                    z[j] = po_ld4_any(a.z, row, a.D, i, a.y_f32);
                }
                ss.x += po_sq(x[j]);
                ss.y += po_sq(z[j]);
            }
            ss = po_sum2(ss, red);
            const float r1 = a.mix / sqrtf(ss.x * inv_n + a.eps), r2 = a.mix / sqrtf(ss.y * inv_n + a.eps);
            ss.x = 0.f;
#pragma unroll
            for (int j = 0; j < V; ++j) {
                const int i = threadIdx.x + j * nt;
                if (i < nvec) {
                    const float4 u = V == 1 ? w1 : po_ld4(a.b1, i), v = V == 1 ? w2 : po_ld4(a.b2, i);
                    x[j].x = x[j].x * r1 * u.x + z[j].x * r2 * v.x; x[j].y = x[j].y * r1 * u.y + z[j].y * r2 * v.y;
                    x[j].z = x[j].z * r1 * u.z + z[j].z * r2 * v.z; x[j].w = x[j].w * r1 * u.w + z[j].w * r2 * v.w;
                }
                ss.x += po_sq(x[j]);
            }
        } else {
            constexpr int PB = V <= 4 ? 4 : 2;                     // parts in flight together
            float self = 0.f;                                      // weight of the identity parts
            for (int p0 = 0; p0 < a.parts; p0 += PB) {
                long src[PB];
                float w[PB];
#pragma unroll
                for (int q = 0; q < PB; ++q) {
                    const long k = row * a.parts + p0 + q;
                    const bool on = p0 + q < a.parts;
                    const bool id = on && a.ids != nullptr && a.ids[k] < 0;
                    w[q] = on && a.wts ? a.wts[k] : 1.f;
                    if (id) self += w[q];
                    src[q] = !on || id ? -1 : a.pos ? (long)a.pos[k] : k;
                }
#pragma unroll
                for (int j = 0; j < V; ++j) {
                    const int i = threadIdx.x + j * nt;
                    float4 t[PB];
#pragma unroll
                    for (int q = 0; q < PB; ++q)
                        t[q] = i < nvec && src[q] >= 0 ? po_ld4_any(a.y, src[q], a.D, i, a.y_f32) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                    for (int q = 0; q < PB; ++q)
                        if (src[q] >= 0) po_axpy(x[j], w[q], t[q]);
                }
            }
#pragma unroll
            for (int j = 0; j < V; ++j) {
                po_axpy(x[j], self, h[j]);
                ss.x += po_sq(x[j]);
            }
        }
        ss = po_sum2(ss, red + 64);
        const float rs = 1.f / sqrtf(ss.x * inv_n + a.eps);
#pragma unroll
        for (int j = 0; j < V; ++j) {
            const int i = threadIdx.x + j * nt;
            if (i >= nvec) continue;
            const float4 w = V == 1 ? wp : po_ld4(a.post, i);
            h[j].x = fmaf(x[j].x * rs, w.x, h[j].x); h[j].y = fmaf(x[j].y * rs, w.y, h[j].y);
            h[j].z = fmaf(x[j].z * rs, w.z, h[j].z); h[j].w = fmaf(x[j].w * rs, w.w, h[j].w);
            reinterpret_cast<float4*>(a.h + row * a.D)[i] = h[j];
        }
    }
    if (a.out == nullptr) return;
    float rs = 1.f;
    if (a.pre != nullptr) {
        float2 ss = make_float2(0.f, 0.f);
#pragma unroll
        for (int j = 0; j < V; ++j) ss.x += po_sq(h[j]);
        rs = 1.f / sqrtf(po_sum2(ss, red + 128).x * inv_n + a.eps);
    }
#pragma unroll
    for (int j = 0; j < V; ++j) {
        const int i = threadIdx.x + j * nt;
        if (i >= nvec) continue;
        float4 o = h[j];
        if (a.pre != nullptr) {
            const float4 w = V == 1 ? wo : po_ld4(a.pre, i);
            o = make_float4(o.x * rs * w.x, o.y * rs * w.y, o.z * rs * w.z, o.w * rs * w.w);
        }
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

extern "C" int tsb_post_norm(const PostNormArgs* args, void* stream) {
    const PostNormArgs& a = *args;
    TSB_CHECK_ARG(a.D > 0 && a.D % 8 == 0 && a.n > 0 && a.n <= a.D && a.parts > 0, "post_norm: bad shape D=%d n=%d parts=%d", a.D, a.n, a.parts);
    TSB_CHECK_ARG(a.y == nullptr || a.post, "post_norm: the norm's weight is missing");
    TSB_CHECK_ARG(a.z == nullptr || (a.y && a.b1 && a.b2 && a.parts == 1 && !a.ids && !a.pos && !a.wts), "post_norm: two branches of one part each");
    TSB_CHECK_ARG(a.pre == nullptr || a.out, "post_norm: the output is missing");
    if (a.rows == 0) return TSB_OK;
    cudaStream_t s = (cudaStream_t)stream;
    const int nvec = a.D / 4;
    const dim3 grid((unsigned)a.rows);
    // few rows (decode): a float4 per thread, for latency; many rows: two or more each
    if (nvec <= 256 || (a.rows < 296 && nvec <= 1024)) {
        TSB_CHECK_CUDA(tsb_launch(post_norm_kernel<1>, grid, dim3((nvec + 31) & ~31), 0, s, a));
    } else {
        TSB_CHECK_ARG(nvec <= 4096, "post_norm: rows of %d columns (limit 16384)", a.D);
        const int v = nvec <= 1024 ? 2 : nvec <= 2048 ? 4 : 8;
        const dim3 block((((nvec + v - 1) / v) + 31) & ~31);
        if (v == 2) TSB_CHECK_CUDA(tsb_launch(post_norm_kernel<2>, grid, block, 0, s, a));
        else if (v == 4) TSB_CHECK_CUDA(tsb_launch(post_norm_kernel<4>, grid, block, 0, s, a));
        else TSB_CHECK_CUDA(tsb_launch(post_norm_kernel<8>, grid, block, 0, s, a));
    }
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}
