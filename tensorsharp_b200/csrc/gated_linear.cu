// Gated linear attention: a memory per head that forgets at a rate of its own in every key channel.  With S [keys, values]:
//
//   w = sigmoid(z + zb)^(1/tau),   z = W2 t                        decay, from the low rank part t of the projection
//   S <- diag(w) S + k v^T,        o = S^T q
//   out = o / rms(o) * norm * silu(g)
//
// Everything here is f32 (the projections may come as bf16).  Key channels are padded with zeros to D (a multiple of 32) and
// value channels to E (16, above 128: 32); zero q, k, v keep the padding of S zero, and the norm divides by the true size.
// The state of a slot is [H][value][key].
//
//   steps, 32-bit models   gla_step_kernel: token by token; a CTA or a cluster of them per (head, sequence), S in registers;
//                          decay map, recurrence, norm and gate in one kernel
//   prompts, bf16 models   gla_chunk_kernel: 16 tokens at a time on the tensor cores, S in accumulator fragments.  A prompt
//                          is cut into segments so that all SMs work: a first launch finds what every segment adds to an
//                          empty memory, gla_fold_kernel turns that into the memory each segment starts from, and a second
//                          launch gives the outputs
//
// Within a chunk, with b_t the sum of log w up to token t (per key channel, all <= 0 and falling):
//   O = (q_t e^(b_t)) S + A V,   A[t][s] = sum_d q_t k_s e^(b_t - b_s)  (s <= t),   S <- e^(b_16) S + (k_s e^(b_16 - b_s))^T V
// No exponent is positive, so a channel may forget as fast as it likes.  Products are mma.sync on split operands, which keeps f32
// accuracy: tf32 in two parts for (q e^b) S, bf16 in three against the values, which are bf16 themselves; accumulation is f32.
#include <cooperative_groups.h>
#include "attn_mma.cuh"
#include "common.cuh"

namespace cg = cooperative_groups;

struct GlaArgs {
    const void* y; long y_s; int y_f32;      // projection rows
    long q, k, v, g, t;                      // first columns of queries, keys (H * D each), values, gate (H * E each), low rank part
    const float* z; long z_s;                // prompts: the decay's projection [T, H * D] without zb
    const void* w2; int w2_f32;              // steps: [H * D, rank]
    const float* zb;                         // [H * D]
    const float* norm_w;                     // [E], for all heads
    float* state; long state_s;              // slot stride
    const int* cu_q; const long* seq_slots;
    float* seg;                              // [B, segs, H, E, D]: what a segment adds, then what it starts from (segs > 1)
    float* seg_w;                            // [B, segs, H, D]: decay over a segment
    float* core;                             // [T, H, E] where a head's values are spread over CTAs
    void* out; long out_s; int out_f32;      // [T, H * E]
    int T, B, H, D, E, e_n, rank, segs, seg_len;
    float eps, q_scale, inv_tau;
};

namespace {
constexpr float GL_LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float gl_ld(const void* p, long i, int f32) {
    return f32 ? reinterpret_cast<const float*>(p)[i] : bf2f(reinterpret_cast<const bf16*>(p)[i]);
}
__device__ __forceinline__ float gl_silu(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float gl_ex2(float x) {
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
    return r;
}
// log2 of sigmoid(z)^(1/tau), k = log2(e) / tau: (min(z, 0) - log(1 + u)) k with u = e^(-|z|) in (0, 1].  log(1 + u) / u is a
// polynomial of degree 9 through the Chebyshev nodes of [0, 1] (relative error below 1.5e-7 in f32): near u = 0, where a channel
// hardly forgets, 1 + u itself would lose what matters.
__device__ __forceinline__ float gl_log2_decay(float z, float k) {
    const float u = gl_ex2(-fabsf(z) * GL_LOG2E);
    float p = -0.00325637846f;
    p = fmaf(p, u, 0.0199071616f);
    p = fmaf(p, u, -0.0570642017f);
    p = fmaf(p, u, 0.106142648f);
    p = fmaf(p, u, -0.153118625f);
    p = fmaf(p, u, 0.196781173f);
    p = fmaf(p, u, -0.249545589f);
    p = fmaf(p, u, 0.333300054f);
    p = fmaf(p, u, -0.499999046f);
    p = fmaf(p, u, 1.f);
    return fmaf(-u, p, fminf(z, 0.f)) * k;
}
__device__ __forceinline__ float gl_sum8(float v) {
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    v += __shfl_xor_sync(0xffffffffu, v, 2);
    return v + __shfl_xor_sync(0xffffffffu, v, 4);
}
// sum of eight products of a weight row's piece with f32 values
__device__ __forceinline__ float gl_dot8(const void* w, long at, int f32, const float* x, float z) {
    const float4 a = *reinterpret_cast<const float4*>(x), b = *reinterpret_cast<const float4*>(x + 4);
    float w8[8];
    if (f32) {
        const float4 c = *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(w) + at);
        const float4 d = *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(w) + at + 4);
        w8[0] = c.x; w8[1] = c.y; w8[2] = c.z; w8[3] = c.w; w8[4] = d.x; w8[5] = d.y; w8[6] = d.z; w8[7] = d.w;
    } else {
        const uint4 c = *reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(w) + at);
        const bf162* h = reinterpret_cast<const bf162*>(&c);
#pragma unroll
        for (int i = 0; i < 4; ++i) { const float2 f = __bfloat1622float2(h[i]); w8[2 * i] = f.x; w8[2 * i + 1] = f.y; }
    }
    z = fmaf(w8[0], a.x, z); z = fmaf(w8[1], a.y, z); z = fmaf(w8[2], a.z, z); z = fmaf(w8[3], a.w, z);
    z = fmaf(w8[4], b.x, z); z = fmaf(w8[5], b.y, z); z = fmaf(w8[6], b.z, z); return fmaf(w8[7], b.w, z);
}
constexpr int STEP_MAX_CL = 8;
}  // namespace

// ------------------------------------------------------------------------------------------
// Steps.  Grid (H * CL, B), clusters of CL CTAs along x; a CTA has eight lanes per value column, `cols` columns; D = 8 * KPL.
// ------------------------------------------------------------------------------------------
template <int KPL>
__global__ void __launch_bounds__(KPL <= 16 ? 1024 : 512) gla_step_kernel(GlaArgs p, int cl, int cols, int w2_staged) {
    constexpr int D = 8 * KPL, NF = KPL / 4;
    extern __shared__ __align__(16) float sm[];
    float* sq = sm;                  // [D]
    float* sk = sq + D;              // [D]
    float* sw = sk + D;              // [D] decay
    float* sv = sw + D;              // [128]
    float* so = sv + 128;            // [32]: sums of squares per warp
    float* ssum = so + 32;           // [2][CL]: every CTA's sum of squares, alternating
    float* st = ssum + 2 * STEP_MAX_CL;      // [rank]
    void* s2 = st + p.rank;
    const int h = blockIdx.x / cl, part = blockIdx.x % cl, b = blockIdx.y, tid = threadIdx.x, nt = blockDim.x, l8 = tid & 7, grp = tid >> 3;
    // The state, the weights and the batch's metadata are not written by the kernel launched directly before (the projection
    // that makes y), and all kernels before that one have ended: they are on their way while the projection still runs.
    const int q0 = p.cu_q[b], n = p.cu_q[b + 1] - q0;
    if (n <= 0) return;                                            // the whole cluster
    if (cl > 1) asm volatile("barrier.cluster.arrive.release;" ::: "memory");      // waited for ahead of the first remote store
    const int c0 = part * cols, mine = min(cols, p.E - c0), col = c0 + grp;
    const bool on = grp < mine;
    float* S = p.state + p.seq_slots[b] * p.state_s + ((long)h * p.E + (on ? col : 0)) * D + 4 * l8;
    float4 s[NF];
#pragma unroll
    for (int i = 0; i < NF; ++i) s[i] = on ? *reinterpret_cast<const float4*>(S + 32 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
    const long hd = (long)h * D, w_at = hd * p.rank;
    if (w2_staged) {
        const int bytes = D * p.rank * (p.w2_f32 ? 4 : 2);
        const char* src = reinterpret_cast<const char*>(p.w2) + w_at * (p.w2_f32 ? 4 : 2);
        for (int i = tid * 16; i < bytes; i += nt * 16) cp_async16(reinterpret_cast<char*>(s2) + i, src + i);
        cp_async_commit();
    }
    const void* w2 = w2_staged ? s2 : p.w2;
    const long w0 = w2_staged ? 0 : w_at;
    const float nw = on ? p.norm_w[col] : 0.f, kd = p.inv_tau * GL_LOG2E;
    pdl_wait();
    pdl_trigger();
    cp_async_wait<0>();
    cg::cluster_group cluster = cg::this_cluster();
    if (cl > 1) asm volatile("barrier.cluster.wait.acquire;" ::: "memory");
    for (int t = q0; t < q0 + n; ++t) {
        const long row = (long)t * p.y_s;
        for (int i = tid; i < p.rank; i += nt) st[i] = gl_ld(p.y, row + p.t + i, p.y_f32);
        for (int d = tid; d < D; d += nt) {
            sq[d] = gl_ld(p.y, row + p.q + hd + d, p.y_f32) * p.q_scale;
            sk[d] = gl_ld(p.y, row + p.k + hd + d, p.y_f32);
        }
        if (tid < mine) sv[tid] = gl_ld(p.y, row + p.v + (long)h * p.E + c0 + tid, p.y_f32);
        const float gate = on && l8 == 0 ? gl_ld(p.y, row + p.g + (long)h * p.E + col, p.y_f32) : 0.f;
        __syncthreads();
        for (int d = grp; d < D; d += nt >> 3) {                   // eight lanes per channel
            float z = 0.f;
            for (int i = 8 * l8; i < p.rank; i += 64) z = gl_dot8(w2, w0 + (long)d * p.rank + i, p.w2_f32, st + i, z);
            z = gl_sum8(z);
            if (l8 == 0) sw[d] = gl_ex2(gl_log2_decay(z + p.zb[hd + d], kd));
        }
        __syncthreads();
        const float v = on ? sv[grp] : 0.f;
        float o = 0.f;
#pragma unroll
        for (int i = 0; i < NF; ++i) {
            const int e = 4 * l8 + 32 * i;
            const float4 k = *reinterpret_cast<const float4*>(sk + e), w = *reinterpret_cast<const float4*>(sw + e);
            const float4 q = *reinterpret_cast<const float4*>(sq + e);
            s[i].x = fmaf(k.x, v, w.x * s[i].x); o = fmaf(s[i].x, q.x, o);
            s[i].y = fmaf(k.y, v, w.y * s[i].y); o = fmaf(s[i].y, q.y, o);
            s[i].z = fmaf(k.z, v, w.z * s[i].z); o = fmaf(s[i].z, q.z, o);
            s[i].w = fmaf(k.w, v, w.w * s[i].w); o = fmaf(s[i].w, q.w, o);
        }
        o = on ? gl_sum8(o) : 0.f;
        const float o2 = warp_sum(l8 == 0 ? o * o : 0.f);
        if ((tid & 31) == 0) so[tid >> 5] = o2;
        __syncthreads();
        float* sums = ssum + (t & 1) * STEP_MAX_CL;
        float ss = 0.f;
        if (cl > 1) {
            // the first warp hands this CTA's sum to every CTA of the cluster: past the barrier each reads its own memory only
            if (tid < 32) {
                const float x = warp_sum(tid < nt >> 5 ? so[tid] : 0.f);
                if (tid < cl) *cluster.map_shared_rank(sums + part, tid) = x;
            }
            asm volatile("barrier.cluster.arrive.release;" ::: "memory");
            if (on && t == q0 + n - 1) {
#pragma unroll
                for (int i = 0; i < NF; ++i) *reinterpret_cast<float4*>(S + 32 * i) = s[i];
            }
            asm volatile("barrier.cluster.wait.acquire;" ::: "memory");
            for (int r = 0; r < cl; ++r) ss += sums[r];
        } else {
            for (int w = 0; w < nt >> 5; ++w) ss += so[w];
            if (on && t == q0 + n - 1) {
#pragma unroll
                for (int i = 0; i < NF; ++i) *reinterpret_cast<float4*>(S + 32 * i) = s[i];
            }
            if (t + 1 < q0 + n) __syncthreads();                   // before the sums are written again
        }
        if (on && l8 == 0) {
            const float r = o / sqrtf(ss / (float)p.e_n + p.eps) * nw * gl_silu(gate);
            const long at = (long)t * p.out_s + (long)h * p.E + col;
            if (p.out_f32) reinterpret_cast<float*>(p.out)[at] = r;
            else reinterpret_cast<bf16*>(p.out)[at] = f2bf(r);
        }
    }
}

// ------------------------------------------------------------------------------------------
// Prompts.  Grid (segments, H * slices, B); a CTA has a warp per 16 value columns (up to 8), rows of y are bf16.
// S^T tile n of a warp: rows = value columns g, g + 8, tile columns 2 t, 2 t + 1; tile 2 i + e, column m stands for key
// 16 i + 2 m + e, so that a thread's accumulators are the next product's operand and its keys are four neighbours.
//
// Running sums start anew in the middle of a chunk: l_s = b_s for its first eight tokens, b_s - b_8 for the others.  Pairs of
// tokens of one half take e^(l_t - l_s) one by one, those across the middle q_t e^(l_t) against k_s e^(b_8 - b_s).
// ------------------------------------------------------------------------------------------
namespace {
constexpr int GC = 16;                                   // tokens per chunk
constexpr int LA_S = 24;                                 // row stride of A

// shared memory: two stages of raw rows (q, k bf16 with padded rows | z f32 | v, g bf16), then the chunk's vectors
template <int D> struct GlaShape {
    static constexpr int RS = D + 16;                    // raw q, k rows (bf16), and rows of all f32 arrays: fragment loads and the
                                                         // loads of different rows at one column are free of bank conflicts
    static constexpr int LK = D + 8;                     // rows of the split k (bf16)
    static constexpr int stage(int es) { return 4 * GC * (RS + D + es); }
    static constexpr int WORK = 4 * (3 * GC * RS + 4 * D + GC * LA_S + 8 * GC + 16) + 2 * 3 * GC * LK;
    static constexpr int bytes(int es) { return 2 * stage(es) + WORK; }
};

__device__ __forceinline__ void gl_split(float x, uint32_t& hi, uint32_t& lo) {      // x = hi + lo up to 2^-21 |x|
    hi = __float_as_uint(x) & 0xffffe000u;
    lo = __float_as_uint(x - __uint_as_float(hi));
}
__device__ __forceinline__ float2 gl_unpack(uint32_t v) { return __bfloat1622float2(*reinterpret_cast<const bf162*>(&v)); }
// two numbers as sums of three bf16 each (all 24 bits)
__device__ __forceinline__ void gl_split3(float x, float y, uint32_t (&o)[3]) {
#pragma unroll
    for (int i = 0; i < 3; ++i) {
        o[i] = pack_bf16(x, y);
        const float2 f = gl_unpack(o[i]);
        x -= f.x;
        y -= f.y;
    }
}
__device__ __forceinline__ float4 gl_bf4(const bf16* p) {
    const uint2 r = *reinterpret_cast<const uint2*>(p);
    const float2 a = gl_unpack(r.x), b = gl_unpack(r.y);
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ float4 gl_f4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 gl_mul(float4 a, float4 b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }
__device__ __forceinline__ float4 gl_ex2(float4 a) { return make_float4(gl_ex2(a.x), gl_ex2(a.y), gl_ex2(a.z), gl_ex2(a.w)); }
__device__ __forceinline__ float4 gl_sub(float4 a, float4 b) { return make_float4(a.x - b.x, a.y - b.y, a.z - b.z, a.w - b.w); }
__device__ __forceinline__ float gl_dot(float4 a, float4 b, float x) {
    x = fmaf(a.x, b.x, x); x = fmaf(a.y, b.y, x); x = fmaf(a.z, b.z, x); return fmaf(a.w, b.w, x);
}
__device__ __forceinline__ void gl_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
}  // namespace

template <int D, bool OUT>
__global__ void __launch_bounds__(256, D <= 128 ? 2 : 1) gla_chunk_kernel(GlaArgs p, int slices) {
    using Z = GlaShape<D>;
    constexpr int NI = D / 16, RS = Z::RS, LK = Z::LK;
    extern __shared__ __align__(16) unsigned char raw[];
    const int es = p.E / slices, h = blockIdx.y / slices, e0 = (blockIdx.y % slices) * es, b = blockIdx.z, sgm = blockIdx.x;
    const int tid = threadIdx.x, nth = blockDim.x, nw = nth >> 5, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    pdl_wait();
    pdl_trigger();
    const int q0 = p.cu_q[b], n_all = p.cu_q[b + 1] - q0;
    const int from = sgm * p.seg_len, n = min(n_all - from, p.seg_len);
    if (n <= 0 || (!OUT && from + p.seg_len >= n_all)) return;        // (nobody starts from what the last segment leaves)
    const bool last = from + p.seg_len >= n_all;
    const int nc = (n + GC - 1) / GC, stage_bytes = Z::stage(es);
    const long tok0 = q0 + from;
    float* sb = reinterpret_cast<float*>(raw + 2 * stage_bytes);     // [16][RS] running sums l of the log2 decays
    float* sq = sb + GC * RS;                                        // [16][RS] q e^b
    float* sp = sq + GC * RS;                                        // [8][RS] q_t e^(l_t) of the second half, [8][RS] k_s e^(b_8 - b_s) of the first
    float* sc = sp + GC * RS;                                        // [D] decay over the chunk
    float* s1 = sc + D;                                              // [D] decay over the first half
    float* s2 = s1 + D;                                              // [D] over the second
    float* zb = s2 + D;                                              // [D]
    float* sa = zb + D;                                              // [16][LA_S]
    float* sn = sa + GC * LA_S;                                      // [8 warps][16]: sums of squares
    unsigned char* pairs = reinterpret_cast<unsigned char*>(sn + 8 * GC);      // [56]: token pairs t > s of a chunk's halves, t * 16 + s
    bf16* sk = reinterpret_cast<bf16*>(sn + 8 * GC + 16);            // [3][16][LK]: k e^(b_16 - b) as a sum of three, key 16 i + 2 m + e in column 16 i + 8 e + m
    const bf16* y = reinterpret_cast<const bf16*>(p.y);

    auto stage = [&](int ch) {
        unsigned char* dst = raw + (ch & 1) * stage_bytes;
        bf16* dq = reinterpret_cast<bf16*>(dst);
        bf16* dk = dq + GC * RS;
        float* dz = reinterpret_cast<float*>(dk + GC * RS);
        bf16* dv = reinterpret_cast<bf16*>(dz + GC * D);
        bf16* dg = dv + GC * es;
        for (int i = tid; i < GC * (D / 8); i += nth) {
            const int r = i / (D / 8), c = (i % (D / 8)) * 8;
            const bool ok = ch * GC + r < n;
            const long row = (tok0 + ch * GC + (ok ? r : 0)) * p.y_s + (long)h * D + c;
            if (ok) {
                if (OUT) cp_async16(dq + r * RS + c, y + row + p.q);
                cp_async16(dk + r * RS + c, y + row + p.k);
            } else {
                *reinterpret_cast<uint4*>(dq + r * RS + c) = make_uint4(0, 0, 0, 0);
                *reinterpret_cast<uint4*>(dk + r * RS + c) = make_uint4(0, 0, 0, 0);
            }
        }
        for (int i = tid; i < GC * (D / 4); i += nth) {
            const int r = i / (D / 4), c = (i % (D / 4)) * 4;
            if (ch * GC + r < n) cp_async16(dz + r * D + c, p.z + (tok0 + ch * GC + r) * p.z_s + (long)h * D + c);
        }
        for (int i = tid; i < GC * (es / 8); i += nth) {
            const int r = i / (es / 8), c = (i % (es / 8)) * 8;
            const bool ok = ch * GC + r < n;
            const long row = (tok0 + ch * GC + (ok ? r : 0)) * p.y_s + (long)h * p.E + e0 + c;
            if (ok) {
                cp_async16(dv + r * es + c, y + row + p.v);
                if (OUT && slices == 1) cp_async16(dg + r * es + c, y + row + p.g);
            } else {
                *reinterpret_cast<uint4*>(dv + r * es + c) = make_uint4(0, 0, 0, 0);
            }
        }
    };
    stage(0);
    cp_async_commit();

    for (int d = tid; d < D; d += nth) zb[d] = p.zb[(long)h * D + d];
    if (OUT) {
        for (int i = tid; i < GC * LA_S; i += nth) sa[i] = 0.f;      // what lies above the diagonal stays zero
        for (int i = tid; i < 56; i += nth) {
            int r = i % 28, x = 1;
            while (r >= x) r -= x++;
            pairs[i] = (unsigned char)((x + 8 * (i / 28)) * 16 + r + 8 * (i / 28));
        }
    } else {
        for (int i = tid; i < 2 * D; i += nth) sq[i] = 0.f;          // here: log2 decay over the segment, in the queries' place
    }
    float s[2 * NI][4];
    const long head = ((long)h * p.E + e0 + warp * 16) * D;          // of this warp's columns in a state
    float* slot = p.state + p.seq_slots[b] * p.state_s + head;
    float* link = p.seg == nullptr ? nullptr : p.seg + ((long)b * p.segs + sgm) * p.H * p.E * D + head;
    const float* S0 = link != nullptr ? link : slot;
#pragma unroll
    for (int i = 0; i < NI; ++i)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const float4 x = OUT ? gl_f4(S0 + (g + 8 * r) * D + 16 * i + 4 * t) : make_float4(0.f, 0.f, 0.f, 0.f);
            s[2 * i][2 * r] = x.x; s[2 * i + 1][2 * r] = x.y; s[2 * i][2 * r + 1] = x.z; s[2 * i + 1][2 * r + 1] = x.w;
        }
    const int ec = warp * 16 + (g & ~1);                             // columns ec, ec + 1, ec + 8, ec + 9 of the results this thread stores
    float2 nw0 = make_float2(0.f, 0.f), nw1 = nw0;
    if (OUT && slices == 1) {
        nw0 = *reinterpret_cast<const float2*>(p.norm_w + ec);
        nw1 = *reinterpret_cast<const float2*>(p.norm_w + ec + 8);
    }
    const float kd = p.inv_tau * GL_LOG2E;

    for (int ch = 0; ch < nc; ++ch) {
        cp_async_wait<0>();
        __syncthreads();                                             // this chunk is here, and everybody is done with the one before
        if (ch + 1 < nc) stage(ch + 1);
        cp_async_commit();
        const unsigned char* src = raw + (ch & 1) * stage_bytes;
        const bf16* rq = reinterpret_cast<const bf16*>(src);
        const bf16* rk = rq + GC * RS;
        const float* rz = reinterpret_cast<const float*>(rk + GC * RS);
        const bf16* rv = reinterpret_cast<const bf16*>(rz + GC * D);
        const bf16* rg = rv + GC * es;
        // ---- log decays and their running sums: a thread has a channel and half of the tokens
        for (int i = tid; i < 2 * D; i += nth) {
            const int d = i % D, r0 = i / D * 8, have = n - ch * GC - r0;
            float x = 0.f;
            const float z0 = zb[d];
#pragma unroll
            for (int r = 0; r < 8; ++r) {
                if (r < have) x += gl_log2_decay(rz[(r0 + r) * D + d] + z0, kd);
                sb[(r0 + r) * RS + d] = x;
            }
            (r0 ? s2 : s1)[d] = gl_ex2(x);
            if (!OUT) sq[i] += x;
        }
        __syncthreads();
        for (int i = tid; i < GC * (D / 4); i += nth) {
            const int r = i / (D / 4), c = (i % (D / 4)) * 4;
            const float4 l = gl_f4(sb + r * RS + c), k = gl_bf4(rk + r * RS + c);
            float4 kw;
            if (r < 8) {
                kw = gl_mul(k, gl_ex2(gl_sub(gl_f4(sb + 7 * RS + c), l)));
                if (OUT) *reinterpret_cast<float4*>(sp + (8 + r) * RS + c) = kw;
                kw = gl_mul(kw, gl_f4(s2 + c));
            } else {
                kw = gl_mul(k, gl_ex2(gl_sub(gl_f4(sb + 15 * RS + c), l)));
            }
            uint32_t k0[3], k1[3];
            gl_split3(kw.x, kw.z, k0);
            gl_split3(kw.y, kw.w, k1);
            bf16* dk = sk + r * LK + (c & ~15) + ((c & 15) >> 1);
#pragma unroll
            for (int x = 0; x < 3; ++x) {
                *reinterpret_cast<uint32_t*>(dk + x * GC * LK) = k0[x];
                *reinterpret_cast<uint32_t*>(dk + x * GC * LK + 8) = k1[x];
            }
            if (OUT) {
                float4 q = gl_bf4(rq + r * RS + c);
                q = gl_mul(make_float4(q.x * p.q_scale, q.y * p.q_scale, q.z * p.q_scale, q.w * p.q_scale), gl_ex2(l));
                if (r >= 8) {
                    *reinterpret_cast<float4*>(sp + (r - 8) * RS + c) = q;
                    q = gl_mul(q, gl_f4(s1 + c));
                }
                *reinterpret_cast<float4*>(sq + r * RS + c) = q;
            }
            if (r == 0) *reinterpret_cast<float4*>(sc + c) = gl_mul(gl_f4(s1 + c), gl_f4(s2 + c));
        }
        if (OUT) {
            // ---- A within the halves: four lanes per pair of tokens, two per token with itself
            for (int i = tid; i < 256; i += nth) {
                float x = 0.f;
                int tt, ss;
                if (i < 224) {
                    tt = pairs[i >> 2] >> 4;
                    ss = pairs[i >> 2] & 15;
                    const int c0 = 4 * (i & 3);
#pragma unroll 2
                    for (int c = c0; c < D; c += 16)
                        x = gl_dot(gl_mul(gl_bf4(rq + tt * RS + c), gl_bf4(rk + ss * RS + c)), gl_ex2(gl_sub(gl_f4(sb + tt * RS + c), gl_f4(sb + ss * RS + c))), x);
                    x += __shfl_xor_sync(0xffffffffu, x, 2);
                } else {
                    tt = ss = (i - 224) >> 1;
#pragma unroll 2
                    for (int c = 4 * (i & 1); c < D; c += 8) x = gl_dot(gl_bf4(rq + tt * RS + c), gl_bf4(rk + tt * RS + c), x);
                }
                x += __shfl_xor_sync(0xffffffffu, x, 1);
                if ((i < 224 ? i & 3 : i & 1) == 0) sa[tt * LA_S + ss] = x * p.q_scale;
            }
        }
        __syncthreads();
        // ---- values of this warp's columns
        uint32_t v[4];
        ldsm_x4_t(v, rv + ((lane & 7) + 8 * (lane >> 4)) * es + warp * 16 + 8 * ((lane >> 3) & 1));
        float o[2][4] = {};
        if (OUT) {
            // ---- A across the middle
            for (int i = tid; i < 256; i += nth) {
                const float* a = sp + (i >> 5) * RS;
                const float* c = sp + (8 + ((i >> 2) & 7)) * RS;
                float x = 0.f;
#pragma unroll 2
                for (int d = 4 * (i & 3); d < D; d += 16) x = gl_dot(gl_f4(a + d), gl_f4(c + d), x);
                x += __shfl_xor_sync(0xffffffffu, x, 1);
                x += __shfl_xor_sync(0xffffffffu, x, 2);
                if ((i & 3) == 0) sa[(8 + (i >> 5)) * LA_S + ((i >> 2) & 7)] = x;
            }
            // ---- O^T [columns][tokens] from the memory, two groups of eight tokens
            float acc[2][2][4] = {};
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const float4 x0 = gl_f4(sq + g * RS + 16 * i + 4 * t), x1 = gl_f4(sq + (g + 8) * RS + 16 * i + 4 * t);
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const float (&m)[4] = s[2 * i + e];
                    uint32_t ah[4], al[4], h0, l0, h1, l1, h2, l2, h3, l3;
                    gl_split(m[0], ah[0], al[0]); gl_split(m[2], ah[1], al[1]); gl_split(m[1], ah[2], al[2]); gl_split(m[3], ah[3], al[3]);
                    gl_split(e ? x0.y : x0.x, h0, l0); gl_split(e ? x0.w : x0.z, h1, l1);
                    gl_split(e ? x1.y : x1.x, h2, l2); gl_split(e ? x1.w : x1.z, h3, l3);
                    gl_mma(acc[0][0], al, h0, h1);
                    gl_mma(acc[1][0], al, h2, h3);
                    gl_mma(o[0], ah, h0, h1);
                    gl_mma(o[1], ah, h2, h3);
                    gl_mma(acc[0][1], ah, l0, l1);
                    gl_mma(acc[1][1], ah, l2, l3);
                }
            }
#pragma unroll
            for (int u = 0; u < 2; ++u)
#pragma unroll
                for (int x = 0; x < 4; ++x) o[u][x] += acc[u][0][x] + acc[u][1][x];
        }
        // ---- S <- e^(b_16) S + (k e^(b_16 - b))^T V
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const float4 w = gl_f4(sc + 16 * i + 4 * t);
            float (&x)[4] = s[2 * i];
            float (&z)[4] = s[2 * i + 1];
            x[0] *= w.x; x[2] *= w.x; x[1] *= w.z; x[3] *= w.z;
            z[0] *= w.y; z[2] *= w.y; z[1] *= w.w; z[3] *= w.w;
        }
        const bf16* kb = sk + ((lane & 7) + 8 * ((lane >> 3) & 1)) * LK + 8 * (lane >> 4);
#pragma unroll
        for (int x = 2; x >= 0; --x)
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                uint32_t k[4];
                ldsm_x4_t(k, kb + x * GC * LK + 16 * i);
                mma_bf16(s[2 * i], v, k[0], k[1]);
                mma_bf16(s[2 * i + 1], v, k[2], k[3]);
            }
        if (OUT) {
            // ---- O^T from the chunk itself
            __syncthreads();
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const float* a = sa + (8 * u + g) * LA_S + 2 * t;
                const float2 x0 = *reinterpret_cast<const float2*>(a), x1 = *reinterpret_cast<const float2*>(a + 8);
                uint32_t a0[3], a1[3];
                gl_split3(x0.x, x0.y, a0);
                gl_split3(x1.x, x1.y, a1);
#pragma unroll
                for (int x = 2; x >= 0; --x) mma_bf16(o[u], v, a0[x], a1[x]);
            }
            if (slices > 1) {
#pragma unroll
                for (int u = 0; u < 2; ++u)
#pragma unroll
                    for (int x = 0; x < 4; ++x) {
                        const int r = ch * GC + 8 * u + 2 * t + (x & 1);
                        if (r < n) p.core[((tok0 + r) * p.H + h) * p.E + e0 + warp * 16 + g + 8 * (x >> 1)] = o[u][x];
                    }
                continue;
            }
            // ---- sums of squares per token (8 u + 2 t + x) over the warp's columns
#pragma unroll
            for (int u = 0; u < 2; ++u)
#pragma unroll
                for (int x = 0; x < 2; ++x) {
                    float q2 = o[u][x] * o[u][x] + o[u][x + 2] * o[u][x + 2];
                    q2 += __shfl_xor_sync(0xffffffffu, q2, 4);
                    q2 += __shfl_xor_sync(0xffffffffu, q2, 8);
                    q2 += __shfl_xor_sync(0xffffffffu, q2, 16);
                    if (g == 0) sn[warp * GC + 8 * u + 2 * t + x] = q2;
                }
            __syncthreads();
            // ---- norm and gate: neighbouring lanes trade tokens for columns
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int odd = g & 1, r = 8 * u + 2 * t + odd;
                const float y0 = __shfl_xor_sync(0xffffffffu, odd ? o[u][0] : o[u][1], 4), y1 = __shfl_xor_sync(0xffffffffu, odd ? o[u][2] : o[u][3], 4);
                float q2 = 0.f;
                for (int w = 0; w < nw; ++w) q2 += sn[w * GC + r];
                if (ch * GC + r >= n) continue;
                const float rs = 1.f / sqrtf(q2 / (float)p.e_n + p.eps);
                const float2 g0 = __bfloat1622float2(*reinterpret_cast<const bf162*>(rg + r * es + ec));
                const float2 g1 = __bfloat1622float2(*reinterpret_cast<const bf162*>(rg + r * es + ec + 8));
                const float a0 = odd ? y0 : o[u][0], a1 = odd ? o[u][1] : y0, b0 = odd ? y1 : o[u][2], b1 = odd ? o[u][3] : y1;
                bf16* out = reinterpret_cast<bf16*>(p.out) + (tok0 + ch * GC + r) * p.out_s + (long)h * p.E + ec;
                *reinterpret_cast<uint32_t*>(out) = pack_bf16(a0 * rs * nw0.x * gl_silu(g0.x), a1 * rs * nw0.y * gl_silu(g0.y));
                *reinterpret_cast<uint32_t*>(out + 8) = pack_bf16(b0 * rs * nw1.x * gl_silu(g1.x), b1 * rs * nw1.y * gl_silu(g1.y));
            }
        }
    }
    float* dst = OUT ? (last ? slot : nullptr) : link;
    if (dst != nullptr) {
#pragma unroll
        for (int i = 0; i < NI; ++i)
#pragma unroll
            for (int r = 0; r < 2; ++r)
                *reinterpret_cast<float4*>(dst + (g + 8 * r) * D + 16 * i + 4 * t) =
                    make_float4(s[2 * i][2 * r], s[2 * i + 1][2 * r], s[2 * i][2 * r + 1], s[2 * i + 1][2 * r + 1]);
    }
    if (!OUT && e0 == 0) {
        __syncthreads();
        float* w = p.seg_w + (((long)b * p.segs + sgm) * p.H + h) * D;
        for (int d = tid; d < D; d += nth) w[d] = gl_ex2(sq[d] + sq[D + d]);
    }
}

// The memory every segment starts from: seg[j] <- S, S <- seg_w[j] S + (what segment j adds).  Grid (pieces of E * D / 4, H, B).
__global__ void __launch_bounds__(256) gla_fold_kernel(GlaArgs p) {
    pdl_wait();
    pdl_trigger();
    const int i = blockIdx.x * 256 + threadIdx.x, h = blockIdx.y, b = blockIdx.z, n = p.cu_q[b + 1] - p.cu_q[b];
    const long block = (long)p.E * p.D;
    if (4L * i >= block || n <= 0) return;
    const int used = (n + p.seg_len - 1) / p.seg_len, d = 4 * i % p.D;
    float4 s = reinterpret_cast<const float4*>(p.state + p.seq_slots[b] * p.state_s + h * block)[i];
    for (int j = 0; j < used; ++j) {
        const long at = ((long)b * p.segs + j) * p.H + h;
        float4* c = reinterpret_cast<float4*>(p.seg + at * block) + i;
        if (j + 1 == used) {
            *c = s;
            break;
        }
        const float4 x = *c, w = *reinterpret_cast<const float4*>(p.seg_w + at * p.D + d);
        *c = s;
        s = make_float4(fmaf(w.x, s.x, x.x), fmaf(w.y, s.y, x.y), fmaf(w.z, s.z, x.z), fmaf(w.w, s.w, x.w));
    }
}

// Norm and gate where a head's values are spread over CTAs: one warp per (token, head).
__global__ void __launch_bounds__(256) gla_finish_kernel(GlaArgs p) {
    pdl_wait();
    pdl_trigger();
    const long id = (long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (id >= (long)p.T * p.H) return;
    const int lane = threadIdx.x & 31;
    const long t = id / p.H, he = id % p.H * p.E;
    float ss = 0.f;
    for (int e = lane; e < p.E; e += 32) { const float x = p.core[id * p.E + e]; ss = fmaf(x, x, ss); }
    const float rs = 1.f / sqrtf(warp_sum(ss) / (float)p.e_n + p.eps);
    for (int e = lane; e < p.E; e += 32) {
        const float r = p.core[id * p.E + e] * rs * p.norm_w[e] * gl_silu(gl_ld(p.y, t * p.y_s + p.g + he + e, p.y_f32));
        if (p.out_f32) reinterpret_cast<float*>(p.out)[t * p.out_s + he + e] = r;
        else reinterpret_cast<bf16*>(p.out)[t * p.out_s + he + e] = f2bf(r);
    }
}

// ------------------------------------------------------------------------------------------
static int gla_check(const GlaArgs& a, const char* what) {
    TSB_CHECK_ARG(a.H > 0 && a.D >= 32 && a.D <= 256 && a.D % 32 == 0 && a.E >= 16 && a.E <= 256 && a.E % (a.E > 128 ? 32 : 16) == 0 && a.e_n > 0 && a.e_n <= a.E,
                  "%s: %d heads of %d / %d (true value size %d)", what, a.H, a.D, a.E, a.e_n);
    TSB_CHECK_ARG(a.B <= 65535 && a.H <= 16384 && a.state_s % 4 == 0 && a.rank >= 0 && a.rank <= 4096, "%s: %d sequences, %d heads, rank %d", what, a.B, a.H, a.rank);
    return TSB_OK;
}

#define GLA_SIZES(X) X(32) X(64) X(96) X(128) X(160) X(192) X(224) X(256)

template <int D>
static int launch_step(const GlaArgs& a, cudaStream_t s) {
    // few heads and sequences: their columns spread over the SMs; many: a CTA takes as many as it may (the decays are found once)
    const int most = D <= 128 ? 128 : 64;
    int cl = (a.E + most - 1) / most;
    while (cl < STEP_MAX_CL && a.E > 32 * cl && (long)a.B * a.H * cl < 148) cl *= 2;
    const int cols = (((a.E + cl - 1) / cl) + 3) & ~3;             // whole warps
    const size_t fixed = sizeof(float) * (3 * D + 128 + 32 + 2 * STEP_MAX_CL + a.rank), w2 = (size_t)D * a.rank * (a.w2_f32 ? 4 : 2);
    const int staged = fixed + w2 <= 48 * 1024;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(a.H * cl, a.B);
    cfg.blockDim = dim3(8 * cols);
    cfg.dynamicSmemBytes = fixed + (staged ? w2 : 0);
    cfg.stream = s;
    cudaLaunchAttribute at[2];
    at[0].id = cudaLaunchAttributeClusterDimension;
    at[0].val.clusterDim.x = cl;
    at[0].val.clusterDim.y = at[0].val.clusterDim.z = 1;
    at[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = at;
    cfg.numAttrs = tsb_pdl_enabled() ? 2 : 1;
    TSB_CHECK_CUDA(cudaLaunchKernelEx(&cfg, gla_step_kernel<D / 8>, a, cl, cols, staged));
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}

extern "C" int tsb_gla_step(const GlaArgs* args, void* stream) {
    const GlaArgs& a = *args;
    const int rc = gla_check(a, "gla_step");
    if (rc != TSB_OK) return rc;
    TSB_CHECK_ARG(a.rank > 0 && a.rank % 8 == 0, "gla_step: rank %d", a.rank);
    if (a.B == 0) return TSB_OK;
    switch (a.D) {
#define X(D) case D: return launch_step<D>(a, (cudaStream_t)stream);
    GLA_SIZES(X)
#undef X
    }
    return TSB_ERR_UNSUPPORTED;
}

template <int D>
static int launch_prompt(const GlaArgs& a, int slices, cudaStream_t s) {
    const int es = a.E / slices, smem = GlaShape<D>::bytes(es), threads = 2 * es;       // a warp per 16 columns
    static bool configured = false;
    if (!configured) {
        TSB_CHECK_CUDA(cudaFuncSetAttribute(gla_chunk_kernel<D, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, GlaShape<D>::bytes(128)));
        TSB_CHECK_CUDA(cudaFuncSetAttribute(gla_chunk_kernel<D, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, GlaShape<D>::bytes(128)));
        configured = true;
    }
    // the chunk kernels are not dependent launches: their long-lived CTAs would take the first places that the kernel ahead
    // leaves, several on one SM with others idle
    if (a.segs > 1) {
        gla_chunk_kernel<D, false><<<dim3(a.segs - 1, a.H * slices, a.B), threads, smem, s>>>(a, slices);
        TSB_CHECK_LAUNCH();
        TSB_CHECK_CUDA(tsb_launch(gla_fold_kernel, dim3((a.E * a.D / 4 + 255) / 256, a.H, a.B), dim3(256), 0, s, a));
    }
    gla_chunk_kernel<D, true><<<dim3(a.segs, a.H * slices, a.B), threads, smem, s>>>(a, slices);
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}

// Recurrence of a packed batch from bf16 projection rows.  `segs` segments of `seg_len` tokens (a multiple of 16) cover the
// longest sequence; seg and seg_w are needed from two on, core where E is above 128.
extern "C" int tsb_gla_prompt(const GlaArgs* args, int max_q, void* stream) {
    GlaArgs a = *args;
    int rc = gla_check(a, "gla_prompt");
    if (rc != TSB_OK) return rc;
    const int slices = a.E > 128 ? 2 : 1;
    TSB_CHECK_ARG(!a.y_f32 && a.z && !a.out_f32, "gla_prompt: bf16 rows and results, f32 decay projection");
    TSB_CHECK_ARG(((a.y_s | a.q | a.k | a.v | a.g | a.out_s) & 7) == 0 && a.z_s % 4 == 0, "gla_prompt: columns are not 16-byte aligned");
    TSB_CHECK_ARG(a.segs > 0 && a.seg_len > 0 && a.seg_len % GC == 0 && (long)a.segs * a.seg_len >= max_q, "gla_prompt: %d segments of %d tokens for %d",
                  a.segs, a.seg_len, max_q);
    TSB_CHECK_ARG((a.segs == 1 || (a.seg && a.seg_w)) && (slices == 1 || a.core), "gla_prompt: missing buffers");
    if (a.B == 0 || a.T == 0) return TSB_OK;
    if (a.segs == 1) a.seg = nullptr;
    cudaStream_t s = (cudaStream_t)stream;
    switch (a.D) {
#define X(D) case D: rc = launch_prompt<D>(a, slices, s); break;
    GLA_SIZES(X)
#undef X
    }
    if (rc != TSB_OK || slices == 1) return rc;
    TSB_CHECK_CUDA(tsb_launch(gla_finish_kernel, dim3((unsigned)(((long)a.T * a.H + 7) / 8)), dim3(256), 0, s, a));
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}
