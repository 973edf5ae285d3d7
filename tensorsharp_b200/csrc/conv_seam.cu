// The seam of a decoder whose sublayers run side by side on one norm of the residual stream, one of them behind a causal
// convolution over time:
//
//   x    = h + y + sum over the parts of w_j p_j      (residual stream, f32; p: the rows a mixture of experts leaves per token)
//   v    = rmsnorm(x) * w                             -> out
//   c_t  = v_t + sum_j taps[j] v_(t - K + 1 + j)      -> conv (per channel; zeros ahead of a sequence's start)
//
// A sequence's last K - 1 values of v are carried in `state` (f32, [K - 1][D] per slot, oldest first).  The new residual goes to
// a buffer of its own (h_out).
//
//   few rows    conv_seam_kernel<CONV>: everything in one kernel.  A block takes up to `span` >= K - 1 consecutive rows of one
//               sequence, computes the K - 1 rows ahead of them again and holds the last K - 1 of v in registers
//   many rows   a block per row for the sum and the norm, which leaves the row's 1 / rms; then seam_conv_kernel, a thread per four
//               channels and run of tokens, makes v again from that and convolves
// Either way the first block or run of a sequence is the only one that reads the slot's old values, and it writes the new ones.
// Rows are padded with zeros to a multiple of 8 columns; the mean of squares runs over the first n.
#include "common.cuh"

struct ConvSeamArgs {
    const float* h;           // [rows, D]
    float* h_out;             // [rows, D] or null (then y and p are null too)
    const void* y;            // [rows, D] f32 or bf16, or null
    const void* p;            // [P, D] f32 or bf16, or null
    const int* pos;           // [rows * parts] row of p per part, or null: row * parts + j
    const float* wts;         // [rows * parts] weight per part, or null: 1
    const float* w;           // [D]
    const float* taps;        // [K][D] or null: no convolution
    float* state;             // slots of stride state_s
    const int* cu_q;          // [B + 1]
    const long* seq_slots;    // [B]
    void* out;                // [rows, D] or null
    void* conv;               // [rows, D] or null
    float* rs;                // [rows]: 1 / rms of every row, where the convolution is a kernel of its own
    long rows, state_s;
    int D, n, B, K, parts, y_f32, p_f32, out_f32, span;
    float eps;
};

namespace {
__device__ __forceinline__ float4 cs_ld4(const float* p, int i) { return reinterpret_cast<const float4*>(p)[i]; }
__device__ __forceinline__ float4 cs_ld4_any(const void* p, long row, int D, int i, int f32) {
    if (f32) return reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p) + row * D)[i];
    const uint2 r = reinterpret_cast<const uint2*>(reinterpret_cast<const bf16*>(p) + row * D)[i];
    const float2 a = __bfloat1622float2(*reinterpret_cast<const bf162*>(&r.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const bf162*>(&r.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void cs_st4(void* p, long row, int D, int i, int f32, float4 o) {
    if (f32) {
        reinterpret_cast<float4*>(reinterpret_cast<float*>(p) + row * D)[i] = o;
    } else {
        uint2 r;
        *reinterpret_cast<bf162*>(&r.x) = __floats2bfloat162_rn(o.x, o.y);
        *reinterpret_cast<bf162*>(&r.y) = __floats2bfloat162_rn(o.z, o.w);
        reinterpret_cast<uint2*>(reinterpret_cast<bf16*>(p) + row * D)[i] = r;
    }
}
__device__ __forceinline__ void cs_axpy(float4& x, float w, float4 t) {
    x.x = fmaf(w, t.x, x.x); x.y = fmaf(w, t.y, x.y); x.z = fmaf(w, t.z, x.z); x.w = fmaf(w, t.w, x.w);
}
__device__ __forceinline__ void cs_fma(float4& x, float4 w, float4 t) {
    x.x = fmaf(w.x, t.x, x.x); x.y = fmaf(w.y, t.y, x.y); x.z = fmaf(w.z, t.z, x.z); x.w = fmaf(w.w, t.w, x.w);
}

// v of one row; `store`: the new residual is written.  `red`: 64 floats, whose halves consecutive calls use in turn.
template <int V>
__device__ __forceinline__ void cs_row(const ConvSeamArgs& a, long row, float4 (&v)[V], const float4& w0, float* red, int& flip, bool store,
                                       float* rms = nullptr) {
    const int nvec = a.D >> 2, nt = blockDim.x;
#pragma unroll
    for (int j = 0; j < V; ++j) {
        const int i = threadIdx.x + j * nt;
        v[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < nvec) {
            v[j] = cs_ld4(a.h + row * a.D, i);
            if (a.y != nullptr) cs_axpy(v[j], 1.f, cs_ld4_any(a.y, row, a.D, i, a.y_f32));
        }
    }
    if (a.p != nullptr) {
        constexpr int PB = V <= 4 ? 4 : 2;                             // parts in flight together
        for (int p0 = 0; p0 < a.parts; p0 += PB) {
            long src[PB];
            float w[PB];
#pragma unroll
            for (int q = 0; q < PB; ++q) {
                const long k = row * a.parts + p0 + q;
                const bool on = p0 + q < a.parts;
                w[q] = on && a.wts ? a.wts[k] : 1.f;
                src[q] = !on ? -1 : a.pos ? (long)a.pos[k] : k;
            }
#pragma unroll
            for (int j = 0; j < V; ++j) {
                const int i = threadIdx.x + j * nt;
                float4 t[PB];
#pragma unroll
                for (int q = 0; q < PB; ++q) t[q] = i < nvec && src[q] >= 0 ? cs_ld4_any(a.p, src[q], a.D, i, a.p_f32) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                for (int q = 0; q < PB; ++q)
                    if (src[q] >= 0) cs_axpy(v[j], w[q], t[q]);
            }
        }
    }
    float q = 0.f;
#pragma unroll
    for (int j = 0; j < V; ++j) {
        const int i = threadIdx.x + j * nt;
        if (store && i < nvec) reinterpret_cast<float4*>(a.h_out + row * a.D)[i] = v[j];
        q += v[j].x * v[j].x + v[j].y * v[j].y + v[j].z * v[j].z + v[j].w * v[j].w;       // padding is zero
    }
    const int lane = threadIdx.x & 31, wp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    q = warp_sum(q);
    if (nw > 1) {
        float* half = red + 32 * flip;
        flip ^= 1;
        if (lane == 0) half[wp] = q;
        __syncthreads();
        q = warp_sum(lane < nw ? half[lane] : 0.f);
    }
    const float rs = 1.f / sqrtf(q / (float)a.n + a.eps);
    if (rms != nullptr && threadIdx.x == 0) *rms = rs;
#pragma unroll
    for (int j = 0; j < V; ++j) {
        const int i = threadIdx.x + j * nt;
        if (i < nvec) {
            const float4 w = V == 1 ? w0 : cs_ld4(a.w, i);
            v[j] = make_float4(v[j].x * rs * w.x, v[j].y * rs * w.y, v[j].z * rs * w.z, v[j].w * rs * w.w);
        }
    }
}
}  // namespace

// V float4s per thread; H = K - 1 rows of history.  CONV false: a block per row, no convolution.
template <int V, int H, bool CONV>
__global__ void __launch_bounds__(V == 1 ? 1024 : 512) conv_seam_kernel(ConvSeamArgs a) {
    __shared__ float red[64];
    const int nvec = a.D >> 2, nt = blockDim.x;
    float4 w0 = make_float4(0.f, 0.f, 0.f, 0.f);
    if (V == 1 && (int)threadIdx.x < nvec) w0 = cs_ld4(a.w, threadIdx.x);
    int flip = 0;
    float4 v[V];
    if (!CONV) {
        pdl_wait();
        pdl_trigger();
        const long row = blockIdx.x;
        cs_row<V>(a, row, v, w0, red, flip, a.h_out != nullptr, a.rs != nullptr ? a.rs + row : nullptr);
#pragma unroll
        for (int j = 0; j < V; ++j) {
            const int i = threadIdx.x + j * nt;
            if (i < nvec && a.out != nullptr) cs_st4(a.out, row, a.D, i, a.out_f32, v[j]);
        }
        return;
    }
    // this block's sequence and rows (the batch's metadata is not written by the kernel launched directly before)
    int b = 0;
    long r0 = 0;
    if (a.rows == a.B) {
        b = blockIdx.x;
        r0 = b;
    } else {
        long before = 0;
        for (;; ++b) {
            if (b == a.B) return;
            const long n = a.cu_q[b + 1] - a.cu_q[b], blocks = (n + a.span - 1) / a.span;
            if ((long)blockIdx.x < before + blocks) break;
            before += blocks;
        }
        r0 = a.cu_q[b] + ((long)blockIdx.x - before) * a.span;
    }
    const long first = a.cu_q[b], end = a.cu_q[b + 1], r1 = min(end, r0 + a.span);
    float* st = a.state + a.seq_slots[b] * a.state_s;
    float4 hist[H > 0 ? H : 1][V], tap0[H + 1];
    if (V == 1 && (int)threadIdx.x < nvec) {
#pragma unroll
        for (int k = 0; k <= H; ++k) tap0[k] = cs_ld4(a.taps + (long)k * a.D, threadIdx.x);
    }
    if (r0 == first) {
#pragma unroll
        for (int k = 0; k < H; ++k)
#pragma unroll
            for (int j = 0; j < V; ++j) {
                const int i = threadIdx.x + j * nt;
                hist[k][j] = i < nvec ? cs_ld4(st + (long)k * a.D, i) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
    }
    pdl_wait();
    pdl_trigger();
    if (r0 != first) {
#pragma unroll
        for (int k = 0; k < H; ++k) cs_row<V>(a, r0 - H + k, hist[k], w0, red, flip, false);
    }
    for (long row = r0; row < r1; ++row) {
        cs_row<V>(a, row, v, w0, red, flip, a.h_out != nullptr);
#pragma unroll
        for (int j = 0; j < V; ++j) {
            const int i = threadIdx.x + j * nt;
            if (i < nvec) {
                if (a.out != nullptr) cs_st4(a.out, row, a.D, i, a.out_f32, v[j]);
                float4 c = v[j];
#pragma unroll
                for (int k = 0; k < H; ++k) cs_fma(c, V == 1 ? tap0[k] : cs_ld4(a.taps + (long)k * a.D, i), hist[k][j]);
                cs_fma(c, V == 1 ? tap0[H] : cs_ld4(a.taps + (long)H * a.D, i), v[j]);
                cs_st4(a.conv, row, a.D, i, a.out_f32, c);
            }
#pragma unroll
            for (int k = 0; k + 1 < H; ++k) hist[k][j] = hist[k + 1][j];
            if (H > 0) hist[H - 1][j] = v[j];
        }
    }
    if (H == 0 || r0 != first) return;
    if (r1 < end) {                                            // the sequence goes on past this block: its last rows once more
#pragma unroll
        for (int k = 0; k < H; ++k)
            if (end - H + k >= r1) {
                cs_row<V>(a, end - H + k, v, w0, red, flip, false);
#pragma unroll
                for (int j = 0; j < V; ++j) {
                    const int i = threadIdx.x + j * nt;
                    if (i < nvec) reinterpret_cast<float4*>(st + (long)k * a.D)[i] = v[j];
                }
            } else {                                           // a row of this block: number end - H + k, the history ends at r1 - 1
                const int at = (int)(end - r1) + k;            // < H
#pragma unroll
                for (int s = 0; s < H; ++s)
                    if (s == at) {
#pragma unroll
                        for (int j = 0; j < V; ++j) {
                            const int i = threadIdx.x + j * nt;
                            if (i < nvec) reinterpret_cast<float4*>(st + (long)k * a.D)[i] = hist[s][j];
                        }
                    }
            }
    } else {
#pragma unroll
        for (int k = 0; k < H; ++k)
#pragma unroll
            for (int j = 0; j < V; ++j) {
                const int i = threadIdx.x + j * nt;
                if (i < nvec) reinterpret_cast<float4*>(st + (long)k * a.D)[i] = hist[k][j];
            }
    }
}

// Grid (runs of `span` tokens, pieces of 512 channels), 128 threads.
template <int H>
__global__ void __launch_bounds__(128) seam_conv_kernel(ConvSeamArgs a) {
    constexpr int U = 4;                                       // rows loaded together
    pdl_wait();
    pdl_trigger();
    const int i = blockIdx.y * 128 + threadIdx.x;
    int b = 0;
    long before = 0;
    for (;; ++b) {
        if (b == a.B) return;
        const long n = a.cu_q[b + 1] - a.cu_q[b], runs = (n + a.span - 1) / a.span;
        if ((long)blockIdx.x < before + runs) break;
        before += runs;
    }
    if (4 * i >= a.D) return;
    const long first = a.cu_q[b], end = a.cu_q[b + 1], r0 = first + ((long)blockIdx.x - before) * a.span, r1 = min(end, r0 + a.span);
    const float* x = a.h_out != nullptr ? a.h_out : a.h;
    float* st = a.state + a.seq_slots[b] * a.state_s;
    const float4 w = cs_ld4(a.w, i);
    auto norm = [&](float4 t, float rs) { return make_float4(t.x * rs * w.x, t.y * rs * w.y, t.z * rs * w.z, t.w * rs * w.w); };
    float4 tap[H + 1], hist[H > 0 ? H : 1];
#pragma unroll
    for (int k = 0; k <= H; ++k) tap[k] = cs_ld4(a.taps + (long)k * a.D, i);
#pragma unroll
    for (int k = 0; k < H; ++k) hist[k] = r0 == first ? cs_ld4(st + (long)k * a.D, i) : norm(cs_ld4(x + (r0 - H + k) * a.D, i), a.rs[r0 - H + k]);
    for (long row = r0; row < r1; row += U) {
        float4 t[U];
        float rs[U];
#pragma unroll
        for (int q = 0; q < U; ++q)
            if (row + q < r1) {
                t[q] = cs_ld4(x + (row + q) * a.D, i);
                rs[q] = a.rs[row + q];
            }
#pragma unroll
        for (int q = 0; q < U; ++q) {
            if (row + q >= r1) break;
            const float4 v = norm(t[q], rs[q]);
            float4 c = v;
#pragma unroll
            for (int k = 0; k < H; ++k) cs_fma(c, tap[k], hist[k]);
            cs_fma(c, tap[H], v);
#pragma unroll
            for (int k = 0; k + 1 < H; ++k) hist[k] = hist[k + 1];
            if (H > 0) hist[H - 1] = v;
            cs_st4(a.conv, row + q, a.D, i, a.out_f32, c);
        }
    }
    if (H == 0 || r0 != first) return;
#pragma unroll
    for (int k = 0; k < H; ++k) {
        const float4 v = r1 < end ? norm(cs_ld4(x + (end - H + k) * a.D, i), a.rs[end - H + k]) : hist[k];
        reinterpret_cast<float4*>(st + (long)k * a.D)[i] = v;
    }
}

template <int V>
static int launch_conv_seam(const ConvSeamArgs& a, dim3 grid, dim3 block, cudaStream_t s) {
    if (a.taps == nullptr) {
        TSB_CHECK_CUDA(tsb_launch(conv_seam_kernel<V, 0, false>, grid, block, 0, s, a));
        return TSB_OK;
    }
    switch (a.K - 1) {
#define X(H) case H: TSB_CHECK_CUDA(tsb_launch(conv_seam_kernel<V, H, true>, grid, block, 0, s, a)); break;
        X(0) X(1) X(2) X(3) X(4) X(5) X(6) X(7)
#undef X
    }
    return TSB_OK;
}

static int conv_seam_rows(const ConvSeamArgs& a, unsigned blocks, cudaStream_t s) {
    const int nvec = a.D / 4;
    const dim3 grid(blocks);
    int rc;
    if (nvec <= 256 || (a.rows < 296 && nvec <= 1024)) {
        rc = launch_conv_seam<1>(a, grid, dim3((nvec + 31) & ~31), s);
    } else {
        TSB_CHECK_ARG(nvec <= 4096, "conv_seam: rows of %d columns (limit 16384)", a.D);
        const int v = nvec <= 1024 ? 2 : nvec <= 2048 ? 4 : 8;
        const dim3 block((((nvec + v - 1) / v) + 31) & ~31);
        rc = v == 2 ? launch_conv_seam<2>(a, grid, block, s) : v == 4 ? launch_conv_seam<4>(a, grid, block, s) : launch_conv_seam<8>(a, grid, block, s);
    }
    if (rc != TSB_OK) return rc;
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}

extern "C" int tsb_conv_seam(const ConvSeamArgs* args, void* stream) {
    ConvSeamArgs a = *args;
    TSB_CHECK_ARG(a.D > 0 && a.D % 8 == 0 && a.n > 0 && a.n <= a.D && a.state_s % 4 == 0, "conv_seam: bad shape D=%d n=%d", a.D, a.n);
    TSB_CHECK_ARG((a.y == nullptr && a.p == nullptr) == (a.h_out == nullptr) && a.h_out != a.h, "conv_seam: the new residual has a buffer of its own");
    TSB_CHECK_ARG(a.p == nullptr || a.parts > 0, "conv_seam: %d parts", a.parts);
    TSB_CHECK_ARG(a.taps == nullptr || (a.K >= 1 && a.K <= 8 && a.conv && a.cu_q && a.seq_slots && a.B > 0 && (a.K == 1 || a.state)),
                  "conv_seam: %d taps (1 to 8), or no state or output for them", a.K);
    if (a.rows == 0) return TSB_OK;
    cudaStream_t s = (cudaStream_t)stream;
    const int nvec = a.D / 4;
    if (a.taps != nullptr && a.rs != nullptr) {
        // many rows: the sum and the norm without the convolution first
        const float* taps = a.taps;
        a.taps = nullptr;
        const int rc = conv_seam_rows(a, (unsigned)a.rows, s);
        if (rc != TSB_OK) return rc;
        a.taps = taps;
        const long per = a.rows * nvec / (148 * 1024);                 // enough threads first, then longer runs
        a.span = per < 4 ? 4 : per > 32 ? 32 : (int)per;
        if (a.span < a.K - 1) a.span = a.K - 1;
        const dim3 grid((unsigned)(a.rows / a.span + a.B), (nvec + 127) / 128);
        switch (a.K - 1) {
#define X(H) case H: TSB_CHECK_CUDA(tsb_launch(seam_conv_kernel<H>, grid, dim3(128), 0, s, a)); break;
            X(0) X(1) X(2) X(3) X(4) X(5) X(6) X(7)
#undef X
        }
        TSB_CHECK_LAUNCH();
        return TSB_OK;
    }
    a.span = a.rows == a.B ? 1 : a.K - 1 > 4 ? a.K - 1 : 4;
    return conv_seam_rows(a, (unsigned)(a.taps == nullptr || a.rows == a.B ? a.rows : a.rows / a.span + a.B), s);
}
