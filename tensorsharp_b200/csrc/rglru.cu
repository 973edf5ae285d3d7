// Real-gated linear recurrent units (Griffin): per channel, with gates r and i from a matrix per block of channels,
//
//   r = sigmoid(Wr u + br),  i = sigmoid(Wi u + bi),  log a = rate r  (rate <= 0)
//   S <- a S + sqrt(1 - a^2) i u,       out = S gelu(y)
//
// Everything here is f32 but the products' inputs in bf16 models.  `u` comes from the short convolution.
//
//   few tokens   rglru_step_kernel: gates, recurrence and output branch in one kernel, token by token
//   prompts      the gates' products run as one grouped matrix product (a group per block), then a scan.  A prompt is cut into
//                segments so that all SMs work: rglru_scan_kernel<false> finds every segment's decay and what it adds to an empty
//                state, rglru_scan_kernel<true> folds those of the segments ahead and gives the outputs
#include "common.cuh"

struct RglruArgs {
    const void* y; long y_s; int y_f32;     // rows whose first W columns are the output branch
    const void* u; int u_f32;               // steps: f32 [T, W]; prompts: [blocks * T, block]
    const void* w; int w_f32;               // steps: [blocks][2 block][block]: rows of Wr, then of Wi
    const float* z;                         // prompts: [blocks * T, 2 block]: Wr u, Wi u
    const float* gate_b;                    // [2][W]
    const float* rate;                      // [W]
    float* state; long state_s;             // [W] per slot
    const int* cu_q; const long* seq_slots;
    float* seg_a;                           // [B][segs][W]: entry j > 0: log decay over segment j - 1
    float* seg_s;                           // [B][segs][W]: entry 0: the state ahead; entry j > 0: what segment j - 1 adds
    void* out; int out_f32;                 // [T, W]
    int T, B, W, block, segs, seg_len;
};

namespace {
constexpr float RG_LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float rg_ld(const void* p, long i, int f32) {
    return f32 ? reinterpret_cast<const float*>(p)[i] : bf2f(reinterpret_cast<const bf16*>(p)[i]);
}
__device__ __forceinline__ float rg_ex2(float x) {
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
    return r;
}
__device__ __forceinline__ float rg_sigmoid(float x) { return __fdividef(1.f, 1.f + rg_ex2(-RG_LOG2E * x)); }
// gelu with the tanh form: 0.5 (1 + tanh(c)) = sigmoid(2 c)
__device__ __forceinline__ float rg_gelu(float x) { return x * rg_sigmoid(1.5957691216057308f * x * fmaf(0.044715f * x, x, 1.f)); }
// a = e^la and sqrt(1 - a^2) for la <= 0.  Near a = 1 the difference would lose what matters: -expm1(t), t = 2 la, by its Taylor series
// (for |t| < 1/4, up to t^7 / 7!: relative error below 1e-8).
__device__ __forceinline__ void rg_decay(float la, float& a, float& mul) {
    a = rg_ex2(la * RG_LOG2E);
    const float t = 2.f * la;
    float p = 1.f / 5040.f;
    p = fmaf(p, t, 1.f / 720.f);
    p = fmaf(p, t, 1.f / 120.f);
    p = fmaf(p, t, 1.f / 24.f);
    p = fmaf(p, t, 1.f / 6.f);
    p = fmaf(p, t, 0.5f);
    p = fmaf(p, t, 1.f);
    mul = sqrtf(t > -0.25f ? -t * p : fmaf(-a, a, 1.f));
}
__device__ __forceinline__ void rg_st(const RglruArgs& a, long at, float v) {
    if (a.out_f32) reinterpret_cast<float*>(a.out)[at] = v;
    else reinterpret_cast<bf16*>(a.out)[at] = f2bf(v);
}
__device__ __forceinline__ float rg_dot8(uint4 w, const float* x, float z) {
    const bf162* h = reinterpret_cast<const bf162*>(&w);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 f = __bfloat1622float2(h[i]);
        z = fmaf(f.x, x[2 * i], z);
        z = fmaf(f.y, x[2 * i + 1], z);
    }
    return z;
}
constexpr int RG_CH = 2;                    // channels per warp
}  // namespace

// Grid (blocks * slices of 16 channels, B), 256 threads; per channel, half a warp has the row of Wr and the other half that of Wi.
__global__ void __launch_bounds__(256) rglru_step_kernel(RglruArgs a) {
    extern __shared__ __align__(16) float su[];             // [block]
    const int slices = (a.block + 8 * RG_CH - 1) / (8 * RG_CH), blk = blockIdx.x / slices, b = blockIdx.y;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, half = lane >> 4, l16 = lane & 15;
    const int c0 = (blockIdx.x % slices) * 8 * RG_CH + warp * RG_CH, bs = a.block;
    // weights, state and metadata are not written by the kernel launched directly before
    const int q0 = a.cu_q[b], n = a.cu_q[b + 1] - q0;
    float* st = a.state + a.seq_slots[b] * a.state_s + (long)blk * bs;
    float s[RG_CH], bias[RG_CH], rate[RG_CH];
    uint4 w0[RG_CH];
    long row[RG_CH];
#pragma unroll
    for (int j = 0; j < RG_CH; ++j) {
        const int c = c0 + j;
        const bool on = c < bs;
        row[j] = ((long)blk * 2 * bs + (long)half * bs + (on ? c : 0)) * bs;
        s[j] = on ? st[c] : 0.f;
        bias[j] = on ? a.gate_b[(long)half * a.W + blk * bs + c] : 0.f;
        rate[j] = on ? a.rate[blk * bs + c] : 0.f;
        w0[j] = make_uint4(0u, 0u, 0u, 0u);
        if (!a.w_f32 && 8 * l16 < bs) w0[j] = *reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(a.w) + row[j] + 8 * l16);
    }
    pdl_wait();
    pdl_trigger();
    for (int t = q0; t < q0 + n; ++t) {
        const float* u = reinterpret_cast<const float*>(a.u) + (long)t * a.W + (long)blk * bs;
        for (int i = threadIdx.x; i < bs; i += 256) su[i] = u[i];
        __syncthreads();
#pragma unroll
        for (int j = 0; j < RG_CH; ++j) {
            float z = 0.f;
            if (!a.w_f32) {
                if (8 * l16 < bs) z = rg_dot8(w0[j], su + 8 * l16, z);
                for (int i = 8 * l16 + 128; i < bs; i += 128)
                    z = rg_dot8(*reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(a.w) + row[j] + i), su + i, z);
            } else {
                for (int i = l16; i < bs; i += 16) z = fmaf(reinterpret_cast<const float*>(a.w)[row[j] + i], su[i], z);
            }
#pragma unroll
            for (int o = 8; o > 0; o >>= 1) z += __shfl_xor_sync(0xffffffffu, z, o);
            const float gate = rg_sigmoid(z + bias[j]), other = __shfl_xor_sync(0xffffffffu, gate, 16);
            if (lane == 0 && c0 + j < bs) {
                float decay, mul;
                rg_decay(rate[j] * gate, decay, mul);
                s[j] = fmaf(decay, s[j], mul * other * su[c0 + j]);
                const long c = (long)blk * bs + c0 + j;
                rg_st(a, (long)t * a.W + c, s[j] * rg_gelu(rg_ld(a.y, (long)t * a.y_s + c, a.y_f32)));
            }
        }
        __syncthreads();
    }
    if (lane == 0 && n > 0) {
#pragma unroll
        for (int j = 0; j < RG_CH; ++j)
            if (c0 + j < bs) st[c0 + j] = s[j];
    }
}

// Grid (channels / 128, segments, B), a thread per channel.
template <bool OUT>
__global__ void __launch_bounds__(128) rglru_scan_kernel(RglruArgs a) {
    pdl_wait();
    pdl_trigger();
    const int c = blockIdx.x * 128 + threadIdx.x, sgm = blockIdx.y, b = blockIdx.z;
    if (c >= a.W) return;
    const int q0 = a.cu_q[b], n_all = a.cu_q[b + 1] - q0, from = sgm * a.seg_len, n = min(a.seg_len, n_all - from);
    if (n_all <= 0) return;
    float* st = a.state + a.seq_slots[b] * a.state_s + c;
    const long seg = ((long)b * a.segs) * a.W + c;
    if (!OUT && sgm == 0) a.seg_s[seg] = *st;
    if (n <= 0 || (!OUT && from + a.seg_len >= n_all)) return;           // (nobody starts from what the last segment leaves)
    const int blk = c / a.block, cb = c % a.block;
    const float br = a.gate_b[c], bi = a.gate_b[a.W + c], rate = a.rate[c];
    const long row0 = (long)blk * a.T + q0 + from;
    const float* z = a.z + row0 * 2 * a.block + cb;
    const long u0 = row0 * a.block + cb;
    float S = 0.f, sum = 0.f;
    if (OUT) {
        if (a.segs == 1) {
            S = *st;
        } else {
            S = a.seg_s[seg];
#pragma unroll 8
            for (int j = 1; j <= sgm; ++j) S = fmaf(rg_ex2(a.seg_a[seg + (long)j * a.W] * RG_LOG2E), S, a.seg_s[seg + (long)j * a.W]);
        }
    }
#pragma unroll 4
    for (int t = 0; t < n; ++t) {
        const float r = rg_sigmoid(z[(long)t * 2 * a.block] + br), i = rg_sigmoid(z[(long)t * 2 * a.block + a.block] + bi);
        const float u = rg_ld(a.u, u0 + (long)t * a.block, a.u_f32);
        const float la = rate * r;
        float decay, mul;
        rg_decay(la, decay, mul);
        S = fmaf(decay, S, mul * i * u);
        if (OUT) {
            const long row = q0 + from + t;
            rg_st(a, row * a.W + c, S * rg_gelu(rg_ld(a.y, row * a.y_s + c, a.y_f32)));
        } else {
            sum += la;
        }
    }
    if (!OUT) {
        a.seg_a[seg + (long)(sgm + 1) * a.W] = sum;
        a.seg_s[seg + (long)(sgm + 1) * a.W] = S;
    } else if (from + a.seg_len >= n_all) {
        *st = S;
    }
}

static int rglru_check(const RglruArgs& a, const char* what) {
    TSB_CHECK_ARG(a.block > 0 && a.block % 8 == 0 && a.W % a.block == 0 && a.B <= 65535, "%s: %d channels in blocks of %d, %d sequences", what, a.W, a.block, a.B);
    return TSB_OK;
}

extern "C" int tsb_rglru_step(const RglruArgs* args, void* stream) {
    const RglruArgs& a = *args;
    const int rc = rglru_check(a, "rglru_step");
    if (rc != TSB_OK) return rc;
    TSB_CHECK_ARG(a.u_f32 && a.block <= 8192, "rglru_step: blocks of %d channels (limit 8192), f32 inputs", a.block);
    if (a.B == 0 || a.T == 0) return TSB_OK;
    const int slices = (a.block + 8 * RG_CH - 1) / (8 * RG_CH);
    TSB_CHECK_CUDA(tsb_launch(rglru_step_kernel, dim3(a.W / a.block * slices, a.B), dim3(256), a.block * sizeof(float), (cudaStream_t)stream, a));
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}

// `segs` segments of `seg_len` tokens cover the longest sequence; seg_a and seg_s are needed from two on.
extern "C" int tsb_rglru_scan(const RglruArgs* args, int max_q, void* stream) {
    const RglruArgs& a = *args;
    const int rc = rglru_check(a, "rglru_scan");
    if (rc != TSB_OK) return rc;
    TSB_CHECK_ARG(a.segs > 0 && a.segs <= 65535 && a.seg_len > 0 && (long)a.segs * a.seg_len >= max_q && (a.segs == 1 || (a.seg_a && a.seg_s)),
                  "rglru_scan: %d segments of %d tokens for %d", a.segs, a.seg_len, max_q);
    if (a.B == 0 || a.T == 0) return TSB_OK;
    cudaStream_t s = (cudaStream_t)stream;
    const unsigned gx = (a.W + 127) / 128;
    if (a.segs > 1) TSB_CHECK_CUDA(tsb_launch(rglru_scan_kernel<false>, dim3(gx, a.segs - 1, a.B), dim3(128), 0, s, a));
    TSB_CHECK_CUDA(tsb_launch(rglru_scan_kernel<true>, dim3(gx, a.segs, a.B), dim3(128), 0, s, a));
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}
