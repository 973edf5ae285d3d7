// Real-gated linear recurrent units (Griffin): per channel, with gates r and i from a matrix per block of channels,
//
//   r = sigmoid(Wr u + br),  i = sigmoid(Wi u + bi),  log a = rate r  (rate <= 0)
//   S <- a S + sqrt(1 - a^2) i u,       out = S gelu(y)
//
// Everything here is f32 but the products' inputs in bf16 models.  `u` comes from the short convolution.
//
//   few tokens   rglru_step_kernel: gates, recurrence and output branch in one kernel, token by token
//   prompts      the gates' products run as one grouped matrix product (a group per block), then a scan.  A prompt is cut into
//                segments so that all SMs work: rglru_scan_kernel without OUT finds every segment's decay and what it adds to an empty
//                state, the one with OUT folds those of the segments ahead and gives the outputs
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
__device__ __forceinline__ float rg_sigmoid(float x) {
    float r;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.f + rg_ex2(-RG_LOG2E * x)));
    return r;
}
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
    asm("sqrt.approx.f32 %0, %1;" : "=f"(mul) : "f"(t > -0.25f ? -t * p : fmaf(-a, a, 1.f)));
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

// Grid (blocks * slices of 16 channels, groups of RG_SEQ sequences), 256 threads.  A group's rows follow one another and are taken
// RG_SEQ at a time.  A warp has two channels; half of it has their rows of Wr and the other half those of Wi.  Of the sixteen sums
// (channel, row) of a half, lane 8 * channel + row ends up with one, so gates, decays and the output branch are found for all of
// them at once.  The same lane holds the state of the group's sequence `row`.
__global__ void __launch_bounds__(256) rglru_step_kernel(RglruArgs a) {
    constexpr int R = RG_SEQ;
    static_assert(R == 8 && RG_CH == 2, "a half warp's lanes are (channel, row)");
    extern __shared__ __align__(16) float su[];             // [R][block]
    const int slices = (a.block + 8 * RG_CH - 1) / (8 * RG_CH), blk = blockIdx.x / slices, b0 = blockIdx.y * RG_SEQ, b1 = min(a.B, b0 + RG_SEQ);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, half = lane >> 4, l16 = lane & 15, ch = l16 & 8, rr = l16 & 7;
    const int c0 = (blockIdx.x % slices) * 8 * RG_CH + warp * RG_CH, bs = a.block, c = c0 + (ch >> 3);
    // weights, state and metadata are not written by the kernel launched directly before
    const int q0 = a.cu_q[b0], q1 = a.cu_q[b1];
    const bool on = c < bs, mine = on && b0 + rr < b1;
    int ends[R];                                            // ends of the group's sequences
#pragma unroll
    for (int i = 0; i < R; ++i) ends[i] = a.cu_q[min(b0 + i + 1, b1)];
    float* st = a.state + (mine ? a.seq_slots[b0 + rr] : 0) * a.state_s + (long)blk * bs;
    float S = mine ? st[c] : 0.f;
    const float bias = on ? a.gate_b[(long)half * a.W + blk * bs + c] : 0.f, rate = on ? a.rate[blk * bs + c] : 0.f;
    uint4 w0[RG_CH];
    long row[RG_CH];
#pragma unroll
    for (int j = 0; j < RG_CH; ++j) {
        row[j] = ((long)blk * 2 * bs + (long)half * bs + (c0 + j < bs ? c0 + j : 0)) * bs;
        w0[j] = make_uint4(0u, 0u, 0u, 0u);
        if (!a.w_f32 && 8 * l16 < bs) w0[j] = *reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(a.w) + row[j] + 8 * l16);
    }
    pdl_wait();
    pdl_trigger();
    const float* u = reinterpret_cast<const float*>(a.u) + (long)blk * bs;
    for (int t0 = q0; t0 < q1; t0 += R) {
        const int rows = min(R, q1 - t0);
        if (t0 > q0) __syncthreads();                       // everybody is done with the rows before
        for (int i = threadIdx.x; i < R * (bs / 4); i += 256) {
            const int r = i / (bs / 4), e = (i % (bs / 4)) * 4;
            *reinterpret_cast<float4*>(su + r * bs + e) =
                r < rows ? *reinterpret_cast<const float4*>(u + (long)(t0 + r) * a.W + e) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
        const bool live = on && rr < rows, writes = live && half == 0;
        const float y = writes ? rg_ld(a.y, (long)(t0 + rr) * a.y_s + blk * bs + c, a.y_f32) : 0.f;
        float z[RG_CH * R];
#pragma unroll
        for (int i = 0; i < RG_CH * R; ++i) z[i] = 0.f;
        __syncthreads();
        if (!a.w_f32) {
            for (int i = 8 * l16; i < bs; i += 128) {
                uint4 w[RG_CH];
#pragma unroll
                for (int j = 0; j < RG_CH; ++j) w[j] = i < 128 ? w0[j] : *reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(a.w) + row[j] + i);
#pragma unroll
                for (int r = 0; r < R; ++r)
                    if (r < rows) {
                        z[r] = rg_dot8(w[0], su + r * bs + i, z[r]);
                        z[R + r] = rg_dot8(w[1], su + r * bs + i, z[R + r]);
                    }
            }
        } else {
            const float* w = reinterpret_cast<const float*>(a.w);
            for (int i = l16; i < bs; i += 16)
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    z[r] = fmaf(w[row[0] + i], su[r * bs + i], z[r]);
                    z[R + r] = fmaf(w[row[1] + i], su[r * bs + i], z[R + r]);
                }
        }
        // sums over the half: in every step a lane keeps one half of its numbers and hands the other to its partner
#pragma unroll
        for (int n = 8; n > 0; n >>= 1)
#pragma unroll
            for (int i = 0; i < 8; ++i)
                if (i < n) {
                    const bool up = l16 & n;
                    const float give = up ? z[i] : z[i + n];
                    z[i] = (up ? z[i + n] : z[i]) + __shfl_xor_sync(0xffffffffu, give, n);
                }
        const float gate = rg_sigmoid(z[0] + bias), other = __shfl_xor_sync(0xffffffffu, gate, 16);
        float decay, mul;
        rg_decay(rate * (half ? other : gate), decay, mul);
        const float add = live ? mul * (half ? gate : other) * su[rr * bs + c] : 0.f;
        int seq = 0;                                        // the row's sequence
#pragma unroll
        for (int i = 0; i < R; ++i) seq += ends[i] <= t0 + rr;
        const int first = __shfl_sync(0xffffffffu, seq, 0);
        float res = 0.f;
        if (__all_sync(0xffffffffu, rr >= rows || seq == first + rr)) {      // one token of each sequence
            res = fmaf(decay, __shfl_sync(0xffffffffu, S, ch | (seq & 7)), add);
            const float mine_now = __shfl_sync(0xffffffffu, res, ch | ((rr - first) & 7));
            if (rr >= first && rr - first < rows) S = mine_now;
        } else {
            for (int r = 0; r < rows; ++r) {
                const int sq = __shfl_sync(0xffffffffu, seq, r);
                const float d = __shfl_sync(0xffffffffu, decay, ch | r), x = __shfl_sync(0xffffffffu, add, ch | r);
                if (rr == sq) S = fmaf(d, S, x);
                const float now = __shfl_sync(0xffffffffu, S, ch | sq);
                if (rr == r) res = now;
            }
        }
        if (writes) rg_st(a, (long)(t0 + rr) * a.W + blk * bs + c, res * rg_gelu(y));
    }
    if (mine && half == 0 && q0 < q1) st[c] = S;
}

// Grid (channels / 128, segments, B), a thread per channel.
template <bool OUT, bool F32>
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
            u[x] = rg_ld(a.u, u0 + t * a.block, F32);
            y[x] = OUT ? rg_ld(a.y, (q0 + from + t) * a.y_s + c, F32) : 0.f;
        }
#pragma unroll
        for (int x = 0; x < U; ++x) {
            if (t0 + x >= n) break;
            const float la = rate * rg_sigmoid(zr[x] + br);
            float decay, mul;
            rg_decay(la, decay, mul);
            S = fmaf(decay, S, mul * rg_sigmoid(zi[x] + bi) * u[x]);
            if (!OUT) sum += la;
            else if (F32) reinterpret_cast<float*>(a.out)[(q0 + from + t0 + x) * (long)a.W + c] = S * rg_gelu(y[x]);
            else reinterpret_cast<bf16*>(a.out)[(q0 + from + t0 + x) * (long)a.W + c] = f2bf(S * rg_gelu(y[x]));
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
    TSB_CHECK_ARG(a.u_f32 && a.block <= 7168, "rglru_step: blocks of %d channels (limit 7168), f32 inputs", a.block);
    if (a.B == 0 || a.T == 0) return TSB_OK;
    const int slices = (a.block + 8 * RG_CH - 1) / (8 * RG_CH);
    if (a.block > 1536) TSB_CHECK_CUDA(cudaFuncSetAttribute(rglru_step_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, RG_SEQ * a.block * (int)sizeof(float)));
    TSB_CHECK_CUDA(tsb_launch(rglru_step_kernel, dim3(a.W / a.block * slices, (a.B + RG_SEQ - 1) / RG_SEQ), dim3(256), RG_SEQ * a.block * sizeof(float),
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
    TSB_CHECK_ARG(a.u_f32 == a.y_f32 && a.u_f32 == a.out_f32, "rglru_scan: inputs and results of one type");
    if (a.B == 0 || a.T == 0) return TSB_OK;
    cudaStream_t s = (cudaStream_t)stream;
    const unsigned gx = (a.W + 127) / 128;
    if (a.segs > 1) {
        if (a.u_f32) TSB_CHECK_CUDA(tsb_launch(rglru_scan_kernel<false, true>, dim3(gx, a.segs - 1, a.B), dim3(128), 0, s, a));
        else TSB_CHECK_CUDA(tsb_launch(rglru_scan_kernel<false, false>, dim3(gx, a.segs - 1, a.B), dim3(128), 0, s, a));
    }
    if (a.u_f32) TSB_CHECK_CUDA(tsb_launch(rglru_scan_kernel<true, true>, dim3(gx, a.segs, a.B), dim3(128), 0, s, a));
    else TSB_CHECK_CUDA(tsb_launch(rglru_scan_kernel<true, false>, dim3(gx, a.segs, a.B), dim3(128), 0, s, a));
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}
