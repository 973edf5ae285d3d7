// The generalized delta rule with a decay and a removal rate per key channel.  Per head, with the state S [keys, values]:
//
//   u = k / sqrt(sum(k^2) + 1e-6)                                  unit key
//   w = exp(-e^(-1/2) sigmoid(z)),  a = sigmoid(a')                decay, removal rate: one per key channel
//   S <- diag(w) S - (a u)(u^T S) + k v^T                          both terms read the old state
//   o = S^T r;   out = o / rms(o) * norm * sigmoid(g)
//
// Every column of S (one value channel) evolves by itself, so a head is spread over groups of eight lanes, each holding
// one or two columns in registers (lane l: keys 4 l + 32 i .. + 3); the only exchange is the sum u^T S over eight lanes.
// Everything here is f32.  Head sizes are padded with zeros to a multiple of 32 (zero r, k, v keep the padding of S zero);
// the norm divides by the true size n.  The state of a slot is [H][value][key].
//
//   short steps (decode)   gdr_short_kernel: one CTA per (head, sequence); decay projection, unit key, recurrence, norm
//                          and gate in one kernel
//   prompts                gdr_prep_kernel: the per-token vectors (u, w, a, r, and v times the key's length);
//                          gdr_scan_kernel: the recurrence, 32 value channels of a head per CTA, tokens staged in shared
//                          memory by cp.async; gdr_finish_kernel: norm and gate
#include "attn_mma.cuh"
#include "common.cuh"

struct GdrArgs {
    const void* y; long y_s; int y_f32;      // rows [r | k | v | a' | g | t]: five parts of H * D, then the decay's low rank part
    const float* z; long z_s;                // prompts: the decay's projection [T, H * D] without w0
    const void* w2; int w2_f32;              // short steps: [H * D, rank], z = w2 tanh(t)
    const float* w0; const float* ab; const float* norm_w;      // [H * D]
    float* state; long state_s;              // slot stride
    const int* cu_q; const long* seq_slots;
    float* pack;                             // [T, H, 5, D]: u | w | a | r | v * |k|
    float* core;                             // [T, H, D]
    void* out; long out_s; int out_f32;      // [T, H * D]
    int T, B, H, D, n, rank;
    float eps;
};

namespace {
constexpr float KEY_EPS = 1e-6f;

__device__ __forceinline__ float gd_ld(const void* p, long i, int f32) {
    return f32 ? reinterpret_cast<const float*>(p)[i] : bf2f(reinterpret_cast<const bf16*>(p)[i]);
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
__device__ __forceinline__ float sum8(float v) {
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    v += __shfl_xor_sync(0xffffffffu, v, 2);
    return v + __shfl_xor_sync(0xffffffffu, v, 4);
}
// two f32 lanes in one 64-bit register
__device__ __forceinline__ uint64_t f2_pack(float x, float y) {
    uint64_t r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(x), "f"(y));
    return r;
}
__device__ __forceinline__ float f2_sum(uint64_t v) {
    float x, y;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(v));
    return x + y;
}
__device__ __forceinline__ uint64_t f2_fma(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ uint64_t f2_mul(uint64_t a, uint64_t b) {
    uint64_t r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
}  // namespace

// ------------------------------------------------------------------------------------------
// Short steps.  Grid (H, B); D = 8 * KPL.  Up to D = 128 a CTA has 8 D threads and the state stays in registers over the
// tokens; above, 512 threads take the columns in turns and read and write the state for every token.
// ------------------------------------------------------------------------------------------
template <int KPL>
__global__ void __launch_bounds__(KPL <= 16 ? 64 * KPL : 512) gdr_short_kernel(GdrArgs p) {
    constexpr int D = 8 * KPL, NT = KPL <= 16 ? 64 * KPL : 512, COLS = NT / 8, PASSES = (D + COLS - 1) / COLS;
    extern __shared__ __align__(16) float sm[];
    float* sk = sm;              // [D] key
    float* sr = sk + D;          // [D] read vector
    float* sa = sr + D;          // [D] removal rate
    float* sw = sa + D;          // [D] decay
    float* sv = sw + D;          // [D] value
    float* so = sv + D;          // [D] read result
    float* st = so + D;          // [rank] tanh of the low rank part
    const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, lane = tid & 31, l8 = tid & 7, col = tid >> 3;
    const long HD = (long)p.H * D, hc = (long)h * D;
    pdl_wait();
    pdl_trigger();
    const int q0 = p.cu_q[b], n = p.cu_q[b + 1] - q0;
    float* S = p.state + p.seq_slots[b] * p.state_s + hc * D;
    float4 s[KPL / 4];
    if (PASSES == 1 && n > 0) {
#pragma unroll
        for (int i = 0; i < KPL / 4; ++i) s[i] = *reinterpret_cast<const float4*>(S + (long)col * D + 4 * l8 + 32 * i);
    }
    for (int t = q0; t < q0 + n; ++t) {
        const long row = (long)t * p.y_s;
        for (int i = tid; i < p.rank; i += NT) st[i] = tanhf(gd_ld(p.y, row + 5 * HD + i, p.y_f32));
        for (int c = tid; c < D; c += NT) {
            sr[c] = gd_ld(p.y, row + hc + c, p.y_f32);
            sk[c] = gd_ld(p.y, row + HD + hc + c, p.y_f32);
            sv[c] = gd_ld(p.y, row + 2 * HD + hc + c, p.y_f32);
            sa[c] = gd_sigmoid(gd_ld(p.y, row + 3 * HD + hc + c, p.y_f32) + p.ab[hc + c]);
        }
        __syncthreads();
        for (int c = col; c < D; c += COLS) {                     // eight lanes per channel
            float z = 0.f;
            const long wr = (hc + c) * p.rank;
            for (int i = l8; i < p.rank; i += 8) z = fmaf(gd_ld(p.w2, wr + i, p.w2_f32), st[i], z);
            z = sum8(z);
            if (l8 == 0) sw[c] = gd_decay(z + p.w0[hc + c]);
        }
        float kk = 0.f;
#pragma unroll
        for (int i = 0; i < D / 32; ++i) { const float v = sk[lane + 32 * i]; kk = fmaf(v, v, kk); }
        const float inv = 1.f / sqrtf(warp_sum(kk) + KEY_EPS);
        __syncthreads();
#pragma unroll 1
        for (int pass = 0; pass < PASSES; ++pass) {
            const int c = col + pass * COLS;
            if (PASSES > 1 && c >= D) break;                      // whole warps: D and COLS are multiples of 4
            float* sp = S + (long)c * D + 4 * l8;
            if (PASSES > 1) {
#pragma unroll
                for (int i = 0; i < KPL / 4; ++i) s[i] = *reinterpret_cast<const float4*>(sp + 32 * i);
            }
            float d = 0.f;
#pragma unroll
            for (int i = 0; i < KPL / 4; ++i) {
                const float4 k = *reinterpret_cast<const float4*>(sk + 4 * l8 + 32 * i);
                d = fmaf(s[i].x, k.x * inv, d); d = fmaf(s[i].y, k.y * inv, d);
                d = fmaf(s[i].z, k.z * inv, d); d = fmaf(s[i].w, k.w * inv, d);
            }
            d = sum8(d);
            const float v = sv[c];
            float o = 0.f;
#pragma unroll
            for (int i = 0; i < KPL / 4; ++i) {
                const int j = 4 * l8 + 32 * i;
                const float4 k = *reinterpret_cast<const float4*>(sk + j), w = *reinterpret_cast<const float4*>(sw + j);
                const float4 a = *reinterpret_cast<const float4*>(sa + j), r = *reinterpret_cast<const float4*>(sr + j);
                s[i].x = fmaf(k.x, fmaf(-a.x * inv, d, v), w.x * s[i].x); o = fmaf(s[i].x, r.x, o);
                s[i].y = fmaf(k.y, fmaf(-a.y * inv, d, v), w.y * s[i].y); o = fmaf(s[i].y, r.y, o);
                s[i].z = fmaf(k.z, fmaf(-a.z * inv, d, v), w.z * s[i].z); o = fmaf(s[i].z, r.z, o);
                s[i].w = fmaf(k.w, fmaf(-a.w * inv, d, v), w.w * s[i].w); o = fmaf(s[i].w, r.w, o);
            }
            o = sum8(o);
            if (l8 == 0) so[c] = o;
            if (PASSES > 1 || t == q0 + n - 1) {
#pragma unroll
                for (int i = 0; i < KPL / 4; ++i) *reinterpret_cast<float4*>(sp + 32 * i) = s[i];
            }
        }
        __syncthreads();
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < D / 32; ++i) { const float v = so[lane + 32 * i]; ss = fmaf(v, v, ss); }
        const float rs = 1.f / sqrtf(warp_sum(ss) / (float)p.n + p.eps);
        for (int c = tid; c < D; c += NT) {
            const float g = gd_sigmoid(gd_ld(p.y, row + 4 * HD + hc + c, p.y_f32));
            gd_st(p.out, (long)t * p.out_s + hc + c, p.out_f32, so[c] * rs * p.norm_w[hc + c] * g);
        }
    }
}

// ------------------------------------------------------------------------------------------
// Prompts
// ------------------------------------------------------------------------------------------
// One warp per (token, head).
__global__ void __launch_bounds__(256) gdr_prep_kernel(GdrArgs p) {
    pdl_wait();
    pdl_trigger();
    const long id = (long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (id >= (long)p.T * p.H) return;
    const int t = (int)(id / p.H), h = (int)(id % p.H), lane = threadIdx.x & 31, D = p.D;
    const long HD = (long)p.H * D, hc = (long)h * D, row = (long)t * p.y_s;
    float k[8], kk = 0.f;                                          // D <= 256
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int c = lane + 32 * i;
        k[i] = c < D ? gd_ld(p.y, row + HD + hc + c, p.y_f32) : 0.f;
        kk = fmaf(k[i], k[i], kk);
    }
    const float len = sqrtf(warp_sum(kk) + KEY_EPS), inv = 1.f / len;
    float* dst = p.pack + id * 5 * D;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int c = lane + 32 * i;
        if (c >= D) break;
        dst[c] = k[i] * inv;
        dst[D + c] = gd_decay(p.z[(long)t * p.z_s + hc + c] + p.w0[hc + c]);
        dst[2 * D + c] = gd_sigmoid(gd_ld(p.y, row + 3 * HD + hc + c, p.y_f32) + p.ab[hc + c]);
        dst[3 * D + c] = gd_ld(p.y, row + hc + c, p.y_f32);
        dst[4 * D + c] = gd_ld(p.y, row + 2 * HD + hc + c, p.y_f32) * len;
    }
}

// Grid (D / (8 NW), H, B), NW warps: a warp holds eight columns of S, two per group of eight lanes.  With k = |k| u the
// update of a column is  S <- w S + u (v |k| - a (u^T S)).  Pairs of keys are multiplied two at a time (f32x2).
template <int KPL, int NW>
__global__ void __launch_bounds__(32 * NW) gdr_scan_kernel(GdrArgs p) {
    constexpr int D = 8 * KPL, COLS = 8 * NW, REC = 4 * D + COLS, CH = 16, NP = KPL / 2;       // NP: pairs of keys per column
    extern __shared__ __align__(16) float sm[];                    // [2][CH][REC]
    const int h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, lane = tid & 31, l8 = lane & 7;
    const int c0 = blockIdx.x * COLS, cl = (tid >> 5) * 8 + (lane >> 3) * 2;                   // this group's first column in the CTA
    pdl_wait();
    pdl_trigger();
    const int q0 = p.cu_q[b], n = p.cu_q[b + 1] - q0;
    if (n <= 0) return;
    float* S = p.state + p.seq_slots[b] * p.state_s + (long)h * D * D;
    uint64_t s[2][NP];
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int i = 0; i < KPL / 4; ++i) {
            const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(S + (long)(c0 + cl + j) * D + 4 * l8 + 32 * i);
            s[j][2 * i] = v.x;
            s[j][2 * i + 1] = v.y;
        }
    auto stage = [&](int t0, int buf) {
        const int m = min(CH, n - t0);
        for (int i = tid; i < m * (REC / 4); i += 32 * NW) {
            const int t = i / (REC / 4), c = (i % (REC / 4)) * 4;
            const float* src = p.pack + ((long)(q0 + t0 + t) * p.H + h) * 5 * D;
            cp_async16(sm + (buf * CH + t) * REC + c, src + (c < 4 * D ? c : c + c0));
        }
        cp_async_commit();
    };
    stage(0, 0);
    for (int t0 = 0, buf = 0; t0 < n; t0 += CH, buf ^= 1) {
        if (t0 + CH < n) {
            stage(t0 + CH, buf ^ 1);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        const int m = min(CH, n - t0);
#pragma unroll 2
        for (int t = 0; t < m; ++t) {
            const float* rec = sm + (buf * CH + t) * REC;
            uint64_t u[NP], d0[2] = {0ull, 0ull}, d1[2] = {0ull, 0ull};
#pragma unroll
            for (int i = 0; i < KPL / 4; ++i) {
                const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(rec + 4 * l8 + 32 * i);
                u[2 * i] = v.x;
                u[2 * i + 1] = v.y;
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    d0[j] = f2_fma(s[j][2 * i], v.x, d0[j]);
                    d1[j] = f2_fma(s[j][2 * i + 1], v.y, d1[j]);
                }
            }
            uint64_t nd[2], vv[2], o0[2] = {0ull, 0ull}, o1[2] = {0ull, 0ull};
            const float2 v2 = *reinterpret_cast<const float2*>(rec + 4 * D + cl);
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const float d = -sum8(f2_sum(d0[j]) + f2_sum(d1[j]));
                nd[j] = f2_pack(d, d);
                vv[j] = j == 0 ? f2_pack(v2.x, v2.x) : f2_pack(v2.y, v2.y);
            }
#pragma unroll
            for (int i = 0; i < KPL / 4; ++i) {
                const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(rec + D + 4 * l8 + 32 * i);
                const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(rec + 2 * D + 4 * l8 + 32 * i);
                const ulonglong2 r = *reinterpret_cast<const ulonglong2*>(rec + 3 * D + 4 * l8 + 32 * i);
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    s[j][2 * i] = f2_fma(u[2 * i], f2_fma(a.x, nd[j], vv[j]), f2_mul(w.x, s[j][2 * i]));
                    s[j][2 * i + 1] = f2_fma(u[2 * i + 1], f2_fma(a.y, nd[j], vv[j]), f2_mul(w.y, s[j][2 * i + 1]));
                    o0[j] = f2_fma(s[j][2 * i], r.x, o0[j]);
                    o1[j] = f2_fma(s[j][2 * i + 1], r.y, o1[j]);
                }
            }
            // both columns' sums in one butterfly: even lanes go on with the first column, odd lanes with the second
            const float oa = f2_sum(o0[0]) + f2_sum(o1[0]), ob = f2_sum(o0[1]) + f2_sum(o1[1]);
            float o = (lane & 1) ? ob : oa;
            o += __shfl_xor_sync(0xffffffffu, (lane & 1) ? oa : ob, 1);
            o += __shfl_xor_sync(0xffffffffu, o, 2);
            o += __shfl_xor_sync(0xffffffffu, o, 4);
            if (l8 < 2) p.core[((long)(q0 + t0 + t) * p.H + h) * D + c0 + cl + l8] = o;
        }
        __syncthreads();                                           // before this buffer is filled again
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int i = 0; i < KPL / 4; ++i)
            *reinterpret_cast<ulonglong2*>(S + (long)(c0 + cl + j) * D + 4 * l8 + 32 * i) = make_ulonglong2(s[j][2 * i], s[j][2 * i + 1]);
}

// One warp per (token, head).
__global__ void __launch_bounds__(256) gdr_finish_kernel(GdrArgs p) {
    pdl_wait();
    pdl_trigger();
    const long id = (long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (id >= (long)p.T * p.H) return;
    const int t = (int)(id / p.H), h = (int)(id % p.H), lane = threadIdx.x & 31, D = p.D;
    const long HD = (long)p.H * D, hc = (long)h * D;
    float o[8], ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int c = lane + 32 * i;
        o[i] = c < D ? p.core[id * D + c] : 0.f;
        ss = fmaf(o[i], o[i], ss);
    }
    const float rs = 1.f / sqrtf(warp_sum(ss) / (float)p.n + p.eps);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int c = lane + 32 * i;
        if (c >= D) break;
        const float g = gd_sigmoid(gd_ld(p.y, (long)t * p.y_s + 4 * HD + hc + c, p.y_f32));
        gd_st(p.out, (long)t * p.out_s + hc + c, p.out_f32, o[i] * rs * p.norm_w[hc + c] * g);
    }
}

// tanh of `cols` columns of rows of y (stride y_s) -> dense rows [T, ld], zero past the columns
__global__ void __launch_bounds__(256) gdr_tanh_kernel(const void* y, long y_s, int y_f32, long off, int T, int cols, int ld, void* out, int out_f32) {
    pdl_wait();
    pdl_trigger();
    const long i = (long)blockIdx.x * 256 + threadIdx.x;
    if (i >= (long)T * ld) return;
    const int t = (int)(i / ld), c = (int)(i % ld);
    gd_st(out, i, out_f32, c < cols ? tanhf(gd_ld(y, (long)t * y_s + off + c, y_f32)) : 0.f);
}

static int gdr_check(const GdrArgs& a, const char* what) {
    TSB_CHECK_ARG(a.H > 0 && a.D >= 32 && a.D <= 256 && a.D % 32 == 0 && a.n > 0 && a.n <= a.D && a.rank >= 0 && a.rank <= 4096,
                  "%s: heads %d of %d (true size %d), rank %d", what, a.H, a.D, a.n, a.rank);
    TSB_CHECK_ARG(a.B <= 65535 && a.H <= 65535 && a.state_s % 4 == 0, "%s: %d sequences, %d heads", what, a.B, a.H);
    return TSB_OK;
}

#define GDR_SIZES(X) X(4) X(8) X(12) X(16) X(20) X(24) X(28) X(32)

extern "C" int tsb_general_delta_short(const GdrArgs* args, void* stream) {
    const GdrArgs& a = *args;
    const int rc = gdr_check(a, "general_delta_short");
    if (rc != TSB_OK) return rc;
    if (a.B == 0) return TSB_OK;
    cudaStream_t s = (cudaStream_t)stream;
    const size_t smem = sizeof(float) * (6 * (size_t)a.D + a.rank);
    switch (a.D / 8) {
#define X(KPL) case KPL: TSB_CHECK_CUDA(tsb_launch(gdr_short_kernel<KPL>, dim3(a.H, a.B), dim3(KPL <= 16 ? 64 * KPL : 512), smem, s, a)); break;
    GDR_SIZES(X)
#undef X
    }
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}

template <int KPL, int NW>
static int launch_scan(const GdrArgs& a, cudaStream_t s) {
    const size_t smem = sizeof(float) * 2 * 16 * (4 * 8 * KPL + 8 * NW);
    static bool configured = false;
    if (!configured) {
        TSB_CHECK_CUDA(cudaFuncSetAttribute(gdr_scan_kernel<KPL, NW>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        configured = true;
    }
    TSB_CHECK_CUDA(tsb_launch(gdr_scan_kernel<KPL, NW>, dim3(a.D / (8 * NW), a.H, a.B), dim3(32 * NW), smem, s, a));
    return TSB_OK;
}

// Recurrence of a packed batch from prepared projections: prep, scan, finish.
extern "C" int tsb_general_delta_prompt(const GdrArgs* args, int warps, void* stream) {
    const GdrArgs& a = *args;
    int rc = gdr_check(a, "general_delta_prompt");
    if (rc != TSB_OK) return rc;
    TSB_CHECK_ARG(a.z && a.pack && a.core && (warps == 2 || warps == 4), "general_delta_prompt: missing buffers, or %d warps", warps);
    if (a.B == 0 || a.T == 0) return TSB_OK;
    cudaStream_t s = (cudaStream_t)stream;
    const dim3 rows((unsigned)(((long)a.T * a.H + 7) / 8));
    TSB_CHECK_CUDA(tsb_launch(gdr_prep_kernel, rows, dim3(256), 0, s, a));
    switch (a.D / 8) {
#define X(KPL) case KPL: rc = warps == 2 ? launch_scan<KPL, 2>(a, s) : launch_scan<KPL, 4>(a, s); break;
    GDR_SIZES(X)
#undef X
    }
    if (rc != TSB_OK) return rc;
    TSB_CHECK_CUDA(tsb_launch(gdr_finish_kernel, rows, dim3(256), 0, s, a));
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}

extern "C" int tsb_tanh_rows(const void* y, long y_s, int y_f32, long off, int T, int cols, int ld, void* out, int out_f32, void* stream) {
    TSB_CHECK_ARG(T >= 0 && cols >= 0 && ld >= cols, "tanh_rows: T=%d cols=%d ld=%d", T, cols, ld);
    const long n = (long)T * ld;
    if (n == 0) return TSB_OK;
    TSB_CHECK_CUDA(tsb_launch(gdr_tanh_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, (cudaStream_t)stream, y, y_s, y_f32, off, T, cols,
                              ld, out, out_f32));
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}
