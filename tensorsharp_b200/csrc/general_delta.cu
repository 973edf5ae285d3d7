// The generalized delta rule with a decay and a removal rate per key channel.  Per head, with the state S [keys, values]:
//
//   u = k / sqrt(sum(k^2) + 1e-6)                                  unit key
//   w = exp(-e^(-1/2) sigmoid(z)),  a = sigmoid(a')                decay, removal rate: one per key channel
//   S <- diag(w) S - (a u)(u^T S) + k v^T                          both terms read the old state
//   o = S^T r;   out = o / rms(o) * norm * sigmoid(g)
//
// Every column of S (one value channel) evolves by itself, so a head is spread over groups of lanes that hold a few columns
// in registers, each lane a share of the keys; the only exchange is the sum u^T S over a group.  Everything here is f32.  Head sizes are padded with zeros to a multiple of 32 (zero r, k, v keep the padding of S zero);
// the norm divides by the true size n.  The state of a slot is [H][value][key].
//
//   short steps (decode)   gdr_short_kernel: one CTA per (head, sequence); decay projection, unit key, recurrence, norm
//                          and gate in one kernel
//   prompts, f32 models    gdr_prep_kernel: the per-token vectors (u, w, a, r, and v times the key's length);
//                          gdr_scan_kernel: the recurrence token by token, tokens staged in shared memory by cp.async;
//                          gdr_finish_kernel: norm and gate
//   prompts, bf16 models   general_delta_chunk.cu: eight tokens at a time on the tensor cores; gdr_finish_kernel
#include "attn_mma.cuh"
#include "common.cuh"
#include "general_delta.cuh"

namespace {
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
// Short steps.  Grid (H, B); D = 8 * KPL.  Up to D = 128 a CTA has 4 D threads, a group of eight lanes holds two columns, and
// the state stays in registers over the tokens; above, 512 threads take the columns in turns and read and write the state
// for every token.
// ------------------------------------------------------------------------------------------
template <int KPL>
constexpr int gdr_short_threads() { return KPL <= 16 ? 32 * KPL : 512; }

template <int KPL>
__global__ void __launch_bounds__(gdr_short_threads<KPL>()) gdr_short_kernel(GdrArgs p) {
    constexpr int D = 8 * KPL, NT = gdr_short_threads<KPL>(), GROUPS = NT / 8, NF = KPL / 4;
    constexpr bool HELD = KPL <= 16;
    constexpr int C = HELD ? 2 : 1, PASSES = HELD ? 1 : (D + GROUPS - 1) / GROUPS;
    extern __shared__ __align__(16) float sm[];
    float* sk = sm;              // [D] key
    float* sr = sk + D;          // [D] read vector
    float* sa = sr + D;          // [D] removal rate
    float* sw = sa + D;          // [D] decay
    float* sv = sw + D;          // [D] value
    float* so = sv + D;          // [D] read result
    float* st = so + D;          // [rank] tanh of the low rank part
    const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, lane = tid & 31, l8 = tid & 7, grp = tid >> 3;
    const long HD = (long)p.H * D, hc = (long)h * D;
    // The state and the batch's metadata are not written by the kernel launched directly before (the projection that makes
    // y), and all kernels before that one have ended: the state is on its way while the projection still runs.
    const int q0 = p.cu_q[b], n = p.cu_q[b + 1] - q0;
    float* S = p.state + p.seq_slots[b] * p.state_s + hc * D + 4 * l8;
    float4 s[C][NF];
    if (HELD && n > 0) {
#pragma unroll
        for (int j = 0; j < C; ++j)
#pragma unroll
            for (int i = 0; i < NF; ++i) s[j][i] = *reinterpret_cast<const float4*>(S + (long)(grp + j * GROUPS) * D + 32 * i);
    }
    pdl_wait();
    pdl_trigger();
    for (int t = q0; t < q0 + n; ++t) {
        const long row = (long)t * p.y_s;
        for (int i = tid; i < p.rank; i += NT) st[i] = tanhf(gd_ld(p.y, row + 5 * HD + i, p.y_f32));
        for (int c = tid; c < D; c += NT) {
            const float r = gd_ld(p.y, row + hc + c, p.y_f32), k = gd_ld(p.y, row + HD + hc + c, p.y_f32);
            const float v = gd_ld(p.y, row + 2 * HD + hc + c, p.y_f32), a = gd_ld(p.y, row + 3 * HD + hc + c, p.y_f32);
            sr[c] = r;
            sk[c] = k;
            sv[c] = v;
            sa[c] = gd_sigmoid(a + p.ab[hc + c]);
        }
        __syncthreads();
        for (int c = grp; c < D; c += GROUPS) {                   // eight lanes per channel
            float z = 0.f;
            const long wr = (hc + c) * p.rank;
            for (int i = l8; i < p.rank; i += 8) z = fmaf(gd_ld(p.w2, wr + i, p.w2_f32), st[i], z);
            z = sum8(z);
            if (l8 == 0) sw[c] = gd_decay(z + p.w0[hc + c]);
        }
        float kk = 0.f;
#pragma unroll
        for (int i = 0; i < D / 32; ++i) { const float v = sk[lane + 32 * i]; kk = fmaf(v, v, kk); }
        const float inv = 1.f / sqrtf(warp_sum(kk) + GDR_KEY_EPS);
        __syncthreads();
#pragma unroll 1
        for (int pass = 0; pass < PASSES; ++pass) {
            const int c0 = grp + pass * GROUPS;
            if (!HELD) {
                if (c0 >= D) break;                               // whole warps: D and GROUPS are multiples of 4
#pragma unroll
                for (int i = 0; i < NF; ++i) s[0][i] = *reinterpret_cast<const float4*>(S + (long)c0 * D + 32 * i);
            }
            float d[C], v[C], o[C];
#pragma unroll
            for (int j = 0; j < C; ++j) { d[j] = o[j] = 0.f; v[j] = sv[c0 + j * GROUPS]; }
#pragma unroll
            for (int i = 0; i < NF; ++i) {
                const float4 k = *reinterpret_cast<const float4*>(sk + 4 * l8 + 32 * i);
#pragma unroll
                for (int j = 0; j < C; ++j) {
                    d[j] = fmaf(s[j][i].x, k.x * inv, d[j]); d[j] = fmaf(s[j][i].y, k.y * inv, d[j]);
                    d[j] = fmaf(s[j][i].z, k.z * inv, d[j]); d[j] = fmaf(s[j][i].w, k.w * inv, d[j]);
                }
            }
#pragma unroll
            for (int j = 0; j < C; ++j) d[j] = sum8(d[j]);
#pragma unroll
            for (int i = 0; i < NF; ++i) {
                const int e = 4 * l8 + 32 * i;
                const float4 k = *reinterpret_cast<const float4*>(sk + e), w = *reinterpret_cast<const float4*>(sw + e);
                const float4 a = *reinterpret_cast<const float4*>(sa + e), r = *reinterpret_cast<const float4*>(sr + e);
                const float4 ai = make_float4(-a.x * inv, -a.y * inv, -a.z * inv, -a.w * inv);
#pragma unroll
                for (int j = 0; j < C; ++j) {
                    float4& x = s[j][i];
                    x.x = fmaf(k.x, fmaf(ai.x, d[j], v[j]), w.x * x.x); o[j] = fmaf(x.x, r.x, o[j]);
                    x.y = fmaf(k.y, fmaf(ai.y, d[j], v[j]), w.y * x.y); o[j] = fmaf(x.y, r.y, o[j]);
                    x.z = fmaf(k.z, fmaf(ai.z, d[j], v[j]), w.z * x.z); o[j] = fmaf(x.z, r.z, o[j]);
                    x.w = fmaf(k.w, fmaf(ai.w, d[j], v[j]), w.w * x.w); o[j] = fmaf(x.w, r.w, o[j]);
                }
            }
#pragma unroll
            for (int j = 0; j < C; ++j) {
                o[j] = sum8(o[j]);
                if (l8 == 0) so[c0 + j * GROUPS] = o[j];
                if (!HELD || t == q0 + n - 1) {
#pragma unroll
                    for (int i = 0; i < NF; ++i) *reinterpret_cast<float4*>(S + (long)(c0 + j * GROUPS) * D + 32 * i) = s[j][i];
                }
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
// One warp per head and PREP_T consecutive tokens; lane l holds channels 4 l + 128 i .. + 3.
constexpr int PREP_T = 4;

template <int NV>
__global__ void __launch_bounds__(256) gdr_prep_kernel(GdrArgs p) {
    pdl_wait();
    pdl_trigger();
    const long id = (long)blockIdx.x * 8 + (threadIdx.x >> 5);
    const int t0 = (int)(id / p.H) * PREP_T, h = (int)(id % p.H), lane = threadIdx.x & 31, D = p.D;
    const long HD = (long)p.H * D, hc = (long)h * D;
    if (t0 >= p.T) {                                               // the last group of warps: the neutral record
        if (id >= (((long)p.T + PREP_T - 1) / PREP_T + 1) * p.H) return;
        float* dst = p.pack + ((long)p.T * p.H + h) * 5 * D;
        for (int c = lane; c < 5 * D; c += 32) dst[c] = c >= D && c < 2 * D ? 1.f : 0.f;
        if (lane < 4) p.link[((long)p.T * p.H + h) * 4 + lane] = 0.f;
        return;
    }
    float u[4 * NV], au[4 * NV];                                   // the previous token's
    const int t1 = min(p.T, t0 + PREP_T + 1);                      // one more for the last token's products with the next key
    for (int t = t0; t < t1; ++t) {
        const long row = (long)t * p.y_s + hc;
        float k[4 * NV], kk = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = 4 * lane + 128 * i;
            const float4 v = c < D ? gd_ld4(p.y, row + HD + c, p.y_f32) : make_float4(0.f, 0.f, 0.f, 0.f);
            k[4 * i] = v.x; k[4 * i + 1] = v.y; k[4 * i + 2] = v.z; k[4 * i + 3] = v.w;
        }
#pragma unroll
        for (int i = 0; i < 4 * NV; ++i) kk = fmaf(k[i], k[i], kk);
        const float len = sqrtf(warp_sum(kk) + GDR_KEY_EPS), inv = 1.f / len;
#pragma unroll
        for (int i = 0; i < 4 * NV; ++i) k[i] *= inv;
        if (t > t0) {
            float g = 0.f, f = 0.f;
#pragma unroll
            for (int i = 0; i < 4 * NV; ++i) { g = fmaf(k[i], au[i], g); f = fmaf(k[i], u[i], f); }
            g = warp_sum(g);
            f = warp_sum(f);
            if (lane == 0) *reinterpret_cast<float4*>(p.link + ((long)(t - 1) * p.H + h) * 4) = make_float4(g, f, 0.f, 0.f);
        }
        if (t == t0 + PREP_T) return;
        if (t == p.T - 1 && lane == 0) *reinterpret_cast<float4*>(p.link + ((long)t * p.H + h) * 4) = make_float4(0.f, 0.f, 0.f, 0.f);
        float* dst = p.pack + ((long)t * p.H + h) * 5 * D;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = 4 * lane + 128 * i;
            if (c < D) {
                const float4 a4 = gd_ld4(p.y, row + 3 * HD + c, p.y_f32), b4 = *reinterpret_cast<const float4*>(p.ab + hc + c);
                const float4 z4 = *reinterpret_cast<const float4*>(p.z + (long)t * p.z_s + hc + c), w4 = *reinterpret_cast<const float4*>(p.w0 + hc + c);
                const float4 r4 = gd_ld4(p.y, row + c, p.y_f32), v4 = gd_ld4(p.y, row + 2 * HD + c, p.y_f32);
                const float4 a = make_float4(gd_sigmoid(a4.x + b4.x), gd_sigmoid(a4.y + b4.y), gd_sigmoid(a4.z + b4.z), gd_sigmoid(a4.w + b4.w));
                *reinterpret_cast<float4*>(dst + c) = make_float4(k[4 * i], k[4 * i + 1], k[4 * i + 2], k[4 * i + 3]);
                *reinterpret_cast<float4*>(dst + D + c) =
                    make_float4(gd_decay(z4.x + w4.x), gd_decay(z4.y + w4.y), gd_decay(z4.z + w4.z), gd_decay(z4.w + w4.w));
                *reinterpret_cast<float4*>(dst + 2 * D + c) = a;
                *reinterpret_cast<float4*>(dst + 3 * D + c) = r4;
                *reinterpret_cast<float4*>(dst + 4 * D + c) = make_float4(v4.x * len, v4.y * len, v4.z * len, v4.w * len);
                au[4 * i] = a.x * k[4 * i]; au[4 * i + 1] = a.y * k[4 * i + 1]; au[4 * i + 2] = a.z * k[4 * i + 2]; au[4 * i + 3] = a.w * k[4 * i + 3];
            } else {
                au[4 * i] = au[4 * i + 1] = au[4 * i + 2] = au[4 * i + 3] = 0.f;
            }
        }
#pragma unroll
        for (int i = 0; i < 4 * NV; ++i) u[i] = k[i];
    }
}

// The recurrence.  A group of G lanes holds C columns of S, lane l the keys 4 l + 4 G i .. + 3 of each; four warps per CTA.
// With k = |k| u the update of a column is  S_t = w S + u (v |k| - a p),  p_t = u_t^T S_(t-1).  The sum over the lanes is kept
// off the path from token to token:
//   p_(t+1) = (u_(t+1) w_t)^T S_(t-1) - (u_(t+1) . a u_t) p_t + (u_(t+1) . u_t) v_t |k_t|
// where the first term is formed one token ahead and the products of neighbouring keys come with the tokens (`link`).  A sum
// over lanes of several columns halves the columns a lane is in charge of while it halves the lanes.  Tokens go in unrolled
// chunks of eight, the last one filled up with tokens that change nothing; the sums for o wait for the chunk's end.  Pairs
// of keys are multiplied two at a time (f32x2).
namespace {
constexpr int SC_CH = 8, SC_ST = 6;              // tokens per chunk, chunks in shared memory

template <int D, int G, int C> struct ScanShape {
    static constexpr int KL = D / G, NP = KL / 2, NF = KL / 4, CPW = C * 32 / G, COLS = 4 * CPW, REC = 4 * D + COLS + 4;
    static constexpr size_t smem = sizeof(float) * SC_ST * SC_CH * REC;
    static_assert(KL % 4 == 0 && D % COLS == 0, "shape");
};

// Sum of q[j] over the group's lanes; every lane gets the sum of one column (scan_owner: which).
template <int G, int C>
__device__ __forceinline__ float scan_sum(float (&q)[C], int l) {
    float x;
    int m = G / 2;
    if (C == 4) {
        const bool hi = l & (G / 2), h2 = l & (G / 4);
        const float a0 = (hi ? q[C - 2] : q[0]) + __shfl_xor_sync(0xffffffffu, hi ? q[0] : q[C - 2], G / 2);
        const float a1 = (hi ? q[C - 1] : q[C > 1]) + __shfl_xor_sync(0xffffffffu, hi ? q[C > 1] : q[C - 1], G / 2);
        x = (h2 ? a1 : a0) + __shfl_xor_sync(0xffffffffu, h2 ? a0 : a1, G / 4);
        m = G / 8;
    } else if (C == 2) {
        const bool hi = l & (G / 2);
        x = (hi ? q[C - 1] : q[0]) + __shfl_xor_sync(0xffffffffu, hi ? q[0] : q[C - 1], G / 2);
        m = G / 4;
    } else {
        x = q[0];
    }
#pragma unroll
    for (int i = G / 2; i >= 1; i >>= 1)
        if (i <= m) x += __shfl_xor_sync(0xffffffffu, x, i);
    return x;
}
template <int G, int C>
__device__ __forceinline__ int scan_owner(int l) { return C == 4 ? ((l & (G / 2)) ? 2 : 0) + ((l & (G / 4)) ? 1 : 0) : C == 2 ? ((l & (G / 2)) ? 1 : 0) : 0; }
// A lane that owns column j
template <int G, int C>
__device__ __forceinline__ int scan_source(int j) { return C == 4 ? (j >> 1) * (G / 2) + (j & 1) * (G / 4) : j * (G / 2); }
}  // namespace

template <int D, int G, int C>
__global__ void __launch_bounds__(128) gdr_scan_kernel(GdrArgs p) {
    using Z = ScanShape<D, G, C>;
    constexpr int NP = Z::NP, NF = Z::NF, COLS = Z::COLS, REC = Z::REC, NV = SC_CH * C;
    extern __shared__ __align__(16) float sm[];                    // [SC_ST * SC_CH][REC]: u | w | a | r | v |k| of the columns | link
    const int h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, lane = tid & 31, l = lane & (G - 1), gb = lane & ~(G - 1);
    const int c0 = blockIdx.x * COLS, cl = (tid >> 5) * Z::CPW + (lane / G) * C;               // this group's first column in the CTA
    pdl_wait();
    pdl_trigger();
    const int q0 = p.cu_q[b], n = p.cu_q[b + 1] - q0;
    if (n <= 0) return;
    float* S = p.state + p.seq_slots[b] * p.state_s + (long)h * D * D;
    const long step = (long)p.H * 5 * D;                           // from token to token
    const float* pk = p.pack + (long)h * 5 * D;
    auto stage = [&](int ch) {                                     // every call commits one group, empty past the end
        const int t0 = ch * SC_CH;
        float* base = sm + (ch % SC_ST) * SC_CH * REC;
        if (t0 < n) {
#pragma unroll
            for (int i = 0; i < SC_CH * D; i += 128) {             // D pieces of 16 bytes per token
                const int e = i + tid, t = e / D, c = (e % D) * 4;
                if (SC_CH * D % 128 == 0 || e < SC_CH * D)
                    cp_async16(base + t * REC + c, pk + (long)(t0 + t < n ? q0 + t0 + t : p.T) * step + c);       // record T changes nothing
            }
            constexpr int VP = COLS / 4 + 1;                       // the columns' values and the link
            for (int e = tid; e < SC_CH * VP; e += 128) {
                const int t = e / VP, c = e % VP;
                const long tok = t0 + t < n ? q0 + t0 + t : p.T;
                float* dst = base + t * REC + 4 * D + c * 4;
                if (c < COLS / 4) cp_async16(dst, pk + tok * step + 4 * D + c0 + c * 4);
                else cp_async16(dst, p.link + (tok * p.H + h) * 4);
            }
        }
        cp_async_commit();
    };
#pragma unroll
    for (int i = 0; i < SC_ST - 1; ++i) stage(i);
    uint64_t s[C][NP], u[NP];
#pragma unroll
    for (int j = 0; j < C; ++j)
#pragma unroll
        for (int i = 0; i < NF; ++i) {
            const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(S + (long)(c0 + cl + j) * D + 4 * l + 4 * G * i);
            s[j][2 * i] = v.x;
            s[j][2 * i + 1] = v.y;
        }
    cp_async_wait<SC_ST - 2>();
    __syncthreads();
#pragma unroll
    for (int i = 0; i < NF; ++i) {
        const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(sm + 4 * l + 4 * G * i);
        u[2 * i] = v.x;
        u[2 * i + 1] = v.y;
    }
    const int own = scan_owner<G, C>(l);
    float pown, pr[C];                                             // p_t of this lane's column, and of all
    {
        float q[C];
#pragma unroll
        for (int j = 0; j < C; ++j) {
            uint64_t d = 0ull;
#pragma unroll
            for (int i = 0; i < NP; ++i) d = f2_fma(s[j][i], u[i], d);
            q[j] = f2_sum(d);
        }
        pown = scan_sum<G, C>(q, l);
#pragma unroll
        for (int j = 0; j < C; ++j) pr[j] = C == 1 ? pown : __shfl_sync(0xffffffffu, pown, gb + scan_source<G, C>(j));
    }
    for (int ch = 0; ch * SC_CH < n; ++ch) {
        stage(ch + SC_ST - 1);
        cp_async_wait<SC_ST - 2>();                                        // the next chunk too: its first key is needed here
        __syncthreads();
        const float* rec0 = sm + (ch % SC_ST) * SC_CH * REC;
        const float* nxt0 = sm + ((ch + 1) % SC_ST) * SC_CH * REC;                             // past the end: not used
        float part[NV];                                            // this lane's share of o: token t, column j at t * C + j
#pragma unroll
        for (int t = 0; t < SC_CH; ++t) {
            const float* rec = rec0 + t * REC;
            const float* key = rec + 4 * l;
            const float* nxt = (t + 1 < SC_CH ? rec + REC : nxt0) + 4 * l;
            const float2 lk = *reinterpret_cast<const float2*>(rec + 4 * D + COLS);
            float v[C], q[C];
            const float vown = rec[4 * D + cl + own];
#pragma unroll
            for (int j = 0; j < C; ++j) v[j] = rec[4 * D + cl + j];
            uint64_t un[NP];
            uint64_t qs[C];
#pragma unroll
            for (int j = 0; j < C; ++j) qs[j] = 0ull;
#pragma unroll
            for (int i = 0; i < NF; ++i) {
                const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(key + D + 4 * G * i);
                const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(nxt + 4 * G * i);
                un[2 * i] = x.x;
                un[2 * i + 1] = x.y;
#pragma unroll
                for (int j = 0; j < C; ++j) {                      // S becomes w S; its product with the next key begins the next p
                    s[j][2 * i] = f2_mul(w.x, s[j][2 * i]);
                    s[j][2 * i + 1] = f2_mul(w.y, s[j][2 * i + 1]);
                    qs[j] = i == 0 ? f2_mul(s[j][2 * i], x.x) : f2_fma(s[j][2 * i], x.x, qs[j]);
                    qs[j] = f2_fma(s[j][2 * i + 1], x.y, qs[j]);
                }
            }
#pragma unroll
            for (int j = 0; j < C; ++j) q[j] = f2_sum(qs[j]);
            const float qown = scan_sum<G, C>(q, l);
            uint64_t os[C];
#pragma unroll
            for (int i = 0; i < NF; ++i) {
                const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(key + 2 * D + 4 * G * i);
                const ulonglong2 r = *reinterpret_cast<const ulonglong2*>(key + 3 * D + 4 * G * i);
#pragma unroll
                for (int j = 0; j < C; ++j) {
                    const uint64_t np = f2_pack(-pr[j], -pr[j]), vv = f2_pack(v[j], v[j]);
                    s[j][2 * i] = f2_fma(u[2 * i], f2_fma(a.x, np, vv), s[j][2 * i]);
                    s[j][2 * i + 1] = f2_fma(u[2 * i + 1], f2_fma(a.y, np, vv), s[j][2 * i + 1]);
                    os[j] = i == 0 ? f2_mul(s[j][2 * i], r.x) : f2_fma(s[j][2 * i], r.x, os[j]);
                    os[j] = f2_fma(s[j][2 * i + 1], r.y, os[j]);
                }
            }
            pown = fmaf(lk.y, vown, fmaf(-lk.x, pown, qown));
#pragma unroll
            for (int j = 0; j < C; ++j) {
                part[t * C + j] = f2_sum(os[j]);
                pr[j] = C == 1 ? pown : __shfl_sync(0xffffffffu, pown, gb + scan_source<G, C>(j));
            }
#pragma unroll
            for (int i = 0; i < NP; ++i) u[i] = un[i];
        }
        int at = 0;                                                // first of the values this lane ends with
#pragma unroll
        for (int m = G / 2, nv = NV; m >= 1; m >>= 1) {
            if (nv > 1) {
                nv >>= 1;
                const bool hi = l & m;
#pragma unroll
                for (int i = 0; i < NV / 2; ++i) {
                    if (i >= nv) break;
                    const float keep = hi ? part[i + nv] : part[i], give = hi ? part[i] : part[i + nv];
                    part[i] = keep + __shfl_xor_sync(0xffffffffu, give, m);
                }
                at += hi ? nv : 0;
            } else {
                part[0] += __shfl_xor_sync(0xffffffffu, part[0], m);
            }
        }
        constexpr int LEFT = NV > G ? NV / G : 1, DUP = G > NV ? G / NV : 1;
        if (DUP == 1 || (l & (DUP - 1)) == 0) {
#pragma unroll
            for (int i = 0; i < LEFT; ++i) {
                const int t = (at + i) / C, j = (at + i) % C;
                if (ch * SC_CH + t < n) p.core[((long)(q0 + ch * SC_CH + t) * p.H + h) * D + c0 + cl + j] = part[i];
            }
        }
        __syncthreads();                                           // before the oldest chunk's place is filled again
    }
    cp_async_wait<0>();
#pragma unroll
    for (int j = 0; j < C; ++j)
#pragma unroll
        for (int i = 0; i < NF; ++i)
            *reinterpret_cast<ulonglong2*>(S + (long)(c0 + cl + j) * D + 4 * l + 4 * G * i) = make_ulonglong2(s[j][2 * i], s[j][2 * i + 1]);
}

// One warp per (token, head).
template <int NV>
__global__ void __launch_bounds__(256) gdr_finish_kernel(GdrArgs p) {
    pdl_wait();
    pdl_trigger();
    const long id = (long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (id >= (long)p.T * p.H) return;
    const int t = (int)(id / p.H), h = (int)(id % p.H), lane = threadIdx.x & 31, D = p.D;
    const long HD = (long)p.H * D, hc = (long)h * D;
    float4 o[NV];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = 4 * lane + 128 * i;
        o[i] = c < D ? *reinterpret_cast<const float4*>(p.core + id * D + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        ss += o[i].x * o[i].x + o[i].y * o[i].y + o[i].z * o[i].z + o[i].w * o[i].w;
    }
    const float rs = 1.f / sqrtf(warp_sum(ss) / (float)p.n + p.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = 4 * lane + 128 * i;
        if (c >= D) break;
        const float4 g = gd_ld4(p.y, (long)t * p.y_s + 4 * HD + hc + c, p.y_f32), w = *reinterpret_cast<const float4*>(p.norm_w + hc + c);
        const float4 v = make_float4(o[i].x * rs * w.x * gd_sigmoid(g.x), o[i].y * rs * w.y * gd_sigmoid(g.y), o[i].z * rs * w.z * gd_sigmoid(g.z),
                                     o[i].w * rs * w.w * gd_sigmoid(g.w));
        const long at = (long)t * p.out_s + hc + c;
        if (p.out_f32) {
            *reinterpret_cast<float4*>(reinterpret_cast<float*>(p.out) + at) = v;
        } else {
            uint2 b;
            *reinterpret_cast<bf162*>(&b.x) = __floats2bfloat162_rn(v.x, v.y);
            *reinterpret_cast<bf162*>(&b.y) = __floats2bfloat162_rn(v.z, v.w);
            *reinterpret_cast<uint2*>(reinterpret_cast<bf16*>(p.out) + at) = b;
        }
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

#define GDR_SIZES(X) X(4) X(8) X(12) X(16) X(20) X(24) X(28) X(32)

extern "C" int tsb_general_delta_short(const GdrArgs* args, void* stream) {
    const GdrArgs& a = *args;
    const int rc = gdr_check(a, "general_delta_short");
    if (rc != TSB_OK) return rc;
    if (a.B == 0) return TSB_OK;
    cudaStream_t s = (cudaStream_t)stream;
    const size_t smem = sizeof(float) * (6 * (size_t)a.D + a.rank);
    switch (a.D / 8) {
#define X(KPL) case KPL: TSB_CHECK_CUDA(tsb_launch(gdr_short_kernel<KPL>, dim3(a.H, a.B), dim3(gdr_short_threads<KPL>()), smem, s, a)); break;
    GDR_SIZES(X)
#undef X
    }
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}

template <int D, int G, int C>
static int launch_scan(const GdrArgs& a, cudaStream_t s) {
    using Z = ScanShape<D, G, C>;
    static bool configured = false;
    if (!configured) {
        TSB_CHECK_CUDA(cudaFuncSetAttribute(gdr_scan_kernel<D, G, C>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)Z::smem));
        configured = true;
    }
    // not as a dependent launch: its long-lived CTAs would take the first places that the other kernel's CTAs leave, several
    // on one SM with others idle
    gdr_scan_kernel<D, G, C><<<dim3(D / Z::COLS, a.H, a.B), 128, Z::smem, s>>>(a);
    return TSB_OK;
}

int tsb_gdr_finish_launch(const GdrArgs& a, cudaStream_t s) {
    const dim3 rows((unsigned)(((long)a.T * a.H + 7) / 8));
    if (a.D <= 128) TSB_CHECK_CUDA(tsb_launch(gdr_finish_kernel<1>, rows, dim3(256), 0, s, a));
    else TSB_CHECK_CUDA(tsb_launch(gdr_finish_kernel<2>, rows, dim3(256), 0, s, a));
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}

// Recurrence of a packed batch from prepared projections: prep, scan (`wide`: twice the columns per group of lanes), finish.
extern "C" int tsb_general_delta_prompt(const GdrArgs* args, int wide, void* stream) {
    const GdrArgs& a = *args;
    int rc = gdr_check(a, "general_delta_prompt");
    if (rc != TSB_OK) return rc;
    TSB_CHECK_ARG(a.z && a.pack && a.link && a.core, "general_delta_prompt: missing buffers");
    TSB_CHECK_ARG(a.y_s % 4 == 0 && a.z_s % 4 == 0 && a.out_s % 4 == 0, "general_delta_prompt: rows of %ld / %ld elements", a.y_s, a.z_s);
    if (a.B == 0 || a.T == 0) return TSB_OK;
    cudaStream_t s = (cudaStream_t)stream;
    const long groups = ((long)a.T + PREP_T - 1) / PREP_T + 1;
    const dim3 prep((unsigned)((groups * a.H + 7) / 8));
    if (a.D <= 128) TSB_CHECK_CUDA(tsb_launch(gdr_prep_kernel<1>, prep, dim3(256), 0, s, a));
    else TSB_CHECK_CUDA(tsb_launch(gdr_prep_kernel<2>, prep, dim3(256), 0, s, a));
    switch (a.D) {
#define X(D, G, C) case D: rc = wide ? launch_scan<D, G, 2 * C>(a, s) : launch_scan<D, G, C>(a, s); break;
    X(32, 8, 1) X(64, 16, 2) X(96, 8, 1) X(128, 32, 2) X(160, 8, 1) X(192, 16, 1) X(224, 8, 1) X(256, 32, 2)
#undef X
    }
    if (rc != TSB_OK) return rc;
    return tsb_gdr_finish_launch(a, s);
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
