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
constexpr int RG_SEQ = 8;                   // sequences per CTA
}  // namespace

// Grid (blocks * slices of 16 channels, groups of RG_SEQ sequences), 256 threads; per channel, half a warp has the row of Wr and the
// other half that of Wi.  A group's rows follow one another; lane i holds the state of the group's sequence i.
__global__ void __launch_bounds__(256) rglru_step_kernel(RglruArgs a) {
    extern __shared__ __align__(16) float su[];             // [2][block]
    const int slices = (a.block + 8 * RG_CH - 1) / (8 * RG_CH), blk = blockIdx.x / slices, b0 = blockIdx.y * RG_SEQ, b1 = min(a.B, b0 + RG_SEQ);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, half = lane >> 4, l16 = lane & 15;
    const int c0 = (blockIdx.x % slices) * 8 * RG_CH + warp * RG_CH, bs = a.block;
    // weights, state and metadata are not written by the kernel launched directly before
    const int q0 = a.cu_q[b0], q1 = a.cu_q[b1];
    const bool mine = b0 + lane < b1;
    const int ends = mine ? a.cu_q[b0 + lane + 1] : q1;
    float* st = a.state + (mine ? a.seq_slots[b0 + lane] : 0) * a.state_s + (long)blk * bs;
    float s[RG_CH], bias[RG_CH], rate[RG_CH];
    uint4 w0[RG_CH];
    long row[RG_CH];
#pragma unroll
    for (int j = 0; j < RG_CH; ++j) {
        const int c = c0 + j;
        const bool on = c < bs;
        row[j] = ((long)blk * 2 * bs + (long)half * bs + (on ? c : 0)) * bs;
        s[j] = on && mine ? st[c] : 0.f;
        bias[j] = on ? a.gate_b[(long)half * a.W + blk * bs + c] : 0.f;
        rate[j] = on ? a.rate[blk * bs + c] : 0.f;
        w0[j] = make_uint4(0u, 0u, 0u, 0u);
        if (!a.w_f32 && 8 * l16 < bs) w0[j] = *reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(a.w) + row[j] + 8 * l16);
    }
    pdl_wait();
    pdl_trigger();
    const float* u = reinterpret_cast<const float*>(a.u) + (long)blk * bs;
    const int yc = blk * bs + c0 + (lane & 1);              // lanes 0 and 1: the output branch of the warp's channels
    auto branch = [&](int t) { return lane < RG_CH && c0 + lane < bs ? rg_ld(a.y, (long)t * a.y_s + yc, a.y_f32) : 0.f; };
    int seq = 0;
    float y = q0 < q1 ? branch(q0) : 0.f;
    if (q0 < q1)
        for (int i = threadIdx.x; i < bs; i += 256) su[i] = u[(long)q0 * a.W + i];
    for (int t = q0; t < q1; ++t) {
        float* cur = su + ((t - q0) & 1) * bs;
        __syncthreads();                                    // this row is here, and everybody is done with the one before
        float y_next = 0.f;
        if (t + 1 < q1) {
            float* nxt = su + ((t + 1 - q0) & 1) * bs;
            for (int i = threadIdx.x; i < bs; i += 256) nxt[i] = u[(long)(t + 1) * a.W + i];
            y_next = branch(t + 1);
        }
        while (__shfl_sync(0xffffffffu, ends, seq) <= t) ++seq;      // (sequences without a token are passed over)
        float res = 0.f;
#pragma unroll
        for (int j = 0; j < RG_CH; ++j) {
            float z = 0.f;
            if (!a.w_f32) {
                if (8 * l16 < bs) z = rg_dot8(w0[j], cur + 8 * l16, z);
                for (int i = 8 * l16 + 128; i < bs; i += 128)
                    z = rg_dot8(*reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(a.w) + row[j] + i), cur + i, z);
            } else {
                for (int i = l16; i < bs; i += 16) z = fmaf(reinterpret_cast<const float*>(a.w)[row[j] + i], cur[i], z);
            }
#pragma unroll
            for (int o = 8; o > 0; o >>= 1) z += __shfl_xor_sync(0xffffffffu, z, o);
            const float gate = rg_sigmoid(z + bias[j]);
            const float r = __shfl_sync(0xffffffffu, gate, 0), i = __shfl_sync(0xffffffffu, gate, 16);
            float decay, mul;
            rg_decay(rate[j] * r, decay, mul);
            const float S = fmaf(decay, __shfl_sync(0xffffffffu, s[j], seq), mul * i * (c0 + j < bs ? cur[c0 + j] : 0.f));
            if (lane == seq) s[j] = S;
            if (lane == j) res = S;
        }
        if (lane < RG_CH && c0 + lane < bs) rg_st(a, (long)t * a.W + yc, res * rg_gelu(y));
        y = y_next;
    }
    if (mine && q0 < q1) {
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
    constexpr int U = 8;                                           // tokens loaded together
    for (int t0 = 0; t0 < n; t0 += U) {
        float zr[U], zi[U], u[U], y[U];
#pragma unroll
        for (int x = 0; x < U; ++x) {
            const long t = min(t0 + x, n - 1);
            zr[x] = z[t * 2 * a.block];
            zi[x] = z[t * 2 * a.block + a.block];
            u[x] = rg_ld(a.u, u0 + t * a.block, a.u_f32);
            y[x] = OUT ? rg_ld(a.y, (q0 + from + t) * a.y_s + c, a.y_f32) : 0.f;
        }
#pragma unroll
        for (int x = 0; x < U; ++x) {
            if (t0 + x >= n) break;
            const float la = rate * rg_sigmoid(zr[x] + br);
            float decay, mul;
            rg_decay(la, decay, mul);
            S = fmaf(decay, S, mul * rg_sigmoid(zi[x] + bi) * u[x]);
            if (OUT) rg_st(a, (q0 + from + t0 + x) * (long)a.W + c, S * rg_gelu(y[x]));
            else sum += la;
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
    TSB_CHECK_ARG(a.u_f32 && a.block <= 4096, "rglru_step: blocks of %d channels (limit 4096), f32 inputs", a.block);
    if (a.B == 0 || a.T == 0) return TSB_OK;
    const int slices = (a.block + 8 * RG_CH - 1) / (8 * RG_CH);
    TSB_CHECK_CUDA(tsb_launch(rglru_step_kernel, dim3(a.W / a.block * slices, (a.B + RG_SEQ - 1) / RG_SEQ), dim3(256), 2 * a.block * sizeof(float),
                              (cudaStream_t)stream, a));
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
