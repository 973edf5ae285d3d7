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
//   steps, 32-bit models   gla_step_kernel: token by token; a cluster of CTAs per (head, sequence), each with up to 32 value
//                          columns in registers; decay map, recurrence, norm and gate in one kernel
//   prompts, bf16 models   gla_chunk_kernel: 16 tokens at a time on the tensor cores, S in accumulator fragments.  A prompt
//                          is cut into segments so that all SMs work: a first launch finds what every segment adds to an
//                          empty memory, gla_fold_kernel turns that into the memory each segment starts from, and a second
//                          launch gives the outputs
//
// Within a chunk, with b_t the sum of log w up to token t (per key channel, all <= 0 and falling):
//   O = (q_t e^(b_t)) S + A V,   A[t][s] = sum_d q_t k_s e^(b_t - b_s)  (s <= t),   S <- e^(b_16) S + (k_s e^(b_16 - b_s))^T V
// No exponent is positive, so a channel may forget as fast as it likes.  Products are mma.sync m16n8k8 on tf32 operands split
// into a high and a low part (values are bf16 and need no split), which keeps f32 accuracy; accumulation is f32.
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
__device__ __forceinline__ float gl_ld(const void* p, long i, int f32) {
    return f32 ? reinterpret_cast<const float*>(p)[i] : bf2f(reinterpret_cast<const bf16*>(p)[i]);
}
__device__ __forceinline__ float gl_silu(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float gl_log_decay(float z, float inv_tau) { return (fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * inv_tau; }
__device__ __forceinline__ float gl_sum8(float v) {
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    v += __shfl_xor_sync(0xffffffffu, v, 2);
    return v + __shfl_xor_sync(0xffffffffu, v, 4);
}
constexpr int STEP_COLS = 32;                // value columns of a CTA of the step kernel, one per group of eight lanes
}  // namespace

// ------------------------------------------------------------------------------------------
// Steps.  Grid (H * CL, B), clusters of CL CTAs along x, 256 threads; D = 8 * KPL.
// ------------------------------------------------------------------------------------------
template <int KPL>
__global__ void __launch_bounds__(256) gla_step_kernel(GlaArgs p, int cl, int cols, int w2_staged) {
    constexpr int D = 8 * KPL, NF = KPL / 4;
    extern __shared__ __align__(16) float sm[];
    float* sq = sm;                  // [D]
    float* sk = sq + D;              // [D]
    float* sw = sk + D;              // [D] decay
    float* sv = sw + D;              // [32]
    float* so = sv + STEP_COLS;      // [32]
    float* ssum = so + STEP_COLS;    // [2]: this CTA's sum of squares, alternating
    float* st = ssum + 4;            // [rank]
    void* s2 = st + ((p.rank + 3) & ~3);
    const int h = blockIdx.x / cl, part = blockIdx.x % cl, b = blockIdx.y, tid = threadIdx.x, l8 = tid & 7, grp = tid >> 3;
    // The state, the weights and the batch's metadata are not written by the kernel launched directly before (the projection
    // that makes y), and all kernels before that one have ended: they are on their way while the projection still runs.
    const int q0 = p.cu_q[b], n = p.cu_q[b + 1] - q0;
    if (n <= 0) return;                                            // the whole cluster
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
        for (int i = tid * 16; i < bytes; i += 256 * 16) cp_async16(reinterpret_cast<char*>(s2) + i, src + i);
        cp_async_commit();
    }
    const void* w2 = w2_staged ? s2 : p.w2;
    const long w0 = w2_staged ? 0 : w_at;
    const float nw = on ? p.norm_w[col] : 0.f;
    pdl_wait();
    pdl_trigger();
    cp_async_wait<0>();
    cg::cluster_group cluster = cg::this_cluster();
    for (int t = q0; t < q0 + n; ++t) {
        const long row = (long)t * p.y_s;
        float* sum = ssum + (t & 1);
        for (int i = tid; i < p.rank; i += 256) st[i] = gl_ld(p.y, row + p.t + i, p.y_f32);
        for (int d = tid; d < D; d += 256) {
            sq[d] = gl_ld(p.y, row + p.q + hd + d, p.y_f32) * p.q_scale;
            sk[d] = gl_ld(p.y, row + p.k + hd + d, p.y_f32);
        }
        if (tid < mine) sv[tid] = gl_ld(p.y, row + p.v + (long)h * p.E + c0 + tid, p.y_f32);
        const float gate = on && l8 == 0 ? gl_ld(p.y, row + p.g + (long)h * p.E + col, p.y_f32) : 0.f;
        __syncthreads();
        for (int d = grp; d < D; d += 32) {                        // eight lanes per channel
            float z = 0.f;
            const long wr = w0 + (long)d * p.rank;
            for (int i = l8; i < p.rank; i += 8) z = fmaf(gl_ld(w2, wr + i, p.w2_f32), st[i], z);
            z = gl_sum8(z);
            if (l8 == 0) sw[d] = expf(gl_log_decay(z + p.zb[hd + d], p.inv_tau));
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
        o = gl_sum8(o);
        if (l8 == 0) so[grp] = on ? o : 0.f;
        __syncthreads();
        if (tid < 32) {
            const float x = so[tid], ss = warp_sum(x * x);
            if (tid == 0) *sum = ss;
        }
        float ss = 0.f;
        if (cl > 1) {
            cluster.sync();                                        // also orders the shared memory of this CTA
            for (int r = 0; r < cl; ++r) ss += *cluster.map_shared_rank(sum, r);
        } else {
            __syncthreads();
            ss = *sum;
        }
        if (on && l8 == 0) {
            const float r = o / sqrtf(ss / (float)p.e_n + p.eps) * nw * gl_silu(gate);
            const long at = (long)t * p.out_s + (long)h * p.E + col;
            if (p.out_f32) reinterpret_cast<float*>(p.out)[at] = r;
            else reinterpret_cast<bf16*>(p.out)[at] = f2bf(r);
        }
    }
    if (on) {
#pragma unroll
        for (int i = 0; i < NF; ++i) *reinterpret_cast<float4*>(S + 32 * i) = s[i];
    }
    if (cl > 1) cluster.sync();                                    // nobody leaves while its sums are still read
}

// ------------------------------------------------------------------------------------------
// Prompts.  Grid (segments, H * slices, B); a CTA has a warp per 16 value columns (up to 8), rows of y are bf16.
// S^T tile n of a warp: rows = value columns g, g + 8, tile columns 2 t, 2 t + 1; tile 2 i + e, column m stands for key
// 16 i + 2 m + e, so that a thread's accumulators are the next product's operand and its keys are four neighbours.
// ------------------------------------------------------------------------------------------
namespace {
constexpr int GC = 16;                                   // tokens per chunk
constexpr int LA_S = 24;                                 // row stride of A

// shared memory (bytes): two stages of raw rows (q, k bf16 | z f32 | v, g bf16), then the chunk's vectors
template <int D> struct GlaShape {
    static constexpr int LQ = D + 16, LK = D + 4;        // row strides of q e^b and k e^(b_16 - b): conflict-free fragment loads
    static constexpr int stage(int es) { return GC * (8 * D + 4 * es); }
    static constexpr int WORK = 4 * (GC * D + GC * LQ + GC * LK + D + GC * LA_S + 8 * GC);
    static constexpr int bytes(int es) { return 2 * stage(es) + WORK; }
};

__device__ __forceinline__ void gl_split(float x, uint32_t& hi, uint32_t& lo) {      // x = hi + lo up to 2^-21 |x|
    hi = __float_as_uint(x) & 0xffffe000u;
    lo = __float_as_uint(x - __uint_as_float(hi));
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
    constexpr int NI = D / 16, LQ = Z::LQ, LK = Z::LK, ND = D / 32;
    constexpr float LOG2E = 1.4426950408889634f;
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
    float* sb = reinterpret_cast<float*>(raw + 2 * stage_bytes);     // [16][D] log decays, then their running sums (log2)
    float* sq = sb + GC * D;                                         // [16][LQ]
    float* sk = sq + GC * LQ;                                        // [16][LK]
    float* sc = sk + GC * LK;                                        // [D] decay over the chunk
    float* sa = sc + D;                                              // [16][LA_S]
    float* sn = sa + GC * LA_S;                                      // [8 warps][16]: sums of squares
    const bf16* y = reinterpret_cast<const bf16*>(p.y);

    auto stage = [&](int ch) {                                       // every call commits one group, empty past the end
        if (ch < nc) {
            unsigned char* dst = raw + (ch & 1) * stage_bytes;
            bf16* dq = reinterpret_cast<bf16*>(dst);
            bf16* dk = dq + GC * D;
            float* dz = reinterpret_cast<float*>(dk + GC * D);
            bf16* dv = reinterpret_cast<bf16*>(dz + GC * D);
            bf16* dg = dv + GC * es;
            for (int i = tid; i < GC * (D / 8); i += nth) {
                const int r = i / (D / 8), c = (i % (D / 8)) * 8;
                const bool ok = ch * GC + r < n;
                const long row = (tok0 + ch * GC + (ok ? r : 0)) * p.y_s + (long)h * D + c;
                if (ok) {
                    if (OUT) cp_async16(dq + r * D + c, y + row + p.q);
                    cp_async16(dk + r * D + c, y + row + p.k);
                } else {
                    *reinterpret_cast<uint4*>(dq + r * D + c) = make_uint4(0, 0, 0, 0);
                    *reinterpret_cast<uint4*>(dk + r * D + c) = make_uint4(0, 0, 0, 0);
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
                    if (OUT) cp_async16(dg + r * es + c, y + row + p.g);
                } else {
                    *reinterpret_cast<uint4*>(dv + r * es + c) = make_uint4(0, 0, 0, 0);
                }
            }
        }
        cp_async_commit();
    };
    stage(0);

    float s[2 * NI][4];
    const long head = ((long)h * p.E + e0 + warp * 16) * D;          // of this warp's columns in a state
    float* slot = p.state + p.seq_slots[b] * p.state_s + head;
    float* link = p.seg == nullptr ? nullptr : p.seg + ((long)b * p.segs + sgm) * p.H * p.E * D + head;
    const float* S0 = link != nullptr ? link : slot;
#pragma unroll
    for (int i = 0; i < NI; ++i)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const float4 x = OUT ? *reinterpret_cast<const float4*>(S0 + (g + 8 * r) * D + 16 * i + 4 * t) : make_float4(0.f, 0.f, 0.f, 0.f);
            s[2 * i][2 * r] = x.x; s[2 * i + 1][2 * r] = x.y; s[2 * i][2 * r + 1] = x.z; s[2 * i + 1][2 * r + 1] = x.w;
        }
    if (!OUT)
        for (int d = tid; d < D; d += nth) sq[d] = 0.f;              // here: log2 decay over the segment, the queries' place
    const float nw0 = OUT && slices == 1 ? p.norm_w[warp * 16 + g] : 0.f, nw1 = OUT && slices == 1 ? p.norm_w[warp * 16 + g + 8] : 0.f;

    for (int ch = 0; ch < nc; ++ch) {
        stage(ch + 1);
        cp_async_wait<1>();
        __syncthreads();
        const unsigned char* src = raw + (ch & 1) * stage_bytes;
        const bf16* rq = reinterpret_cast<const bf16*>(src);
        const bf16* rk = rq + GC * D;
        const float* rz = reinterpret_cast<const float*>(rk + GC * D);
        const bf16* rv = reinterpret_cast<const bf16*>(rz + GC * D);
        bf16* rg = const_cast<bf16*>(rv) + GC * es;
        // ---- log decays, their running sums, what survives the chunk
        for (int i = tid; i < GC * D; i += nth) {
            const int r = i / D, d = i % D;
            sb[i] = ch * GC + r < n ? gl_log_decay(rz[i] + p.zb[(long)h * D + d], p.inv_tau * LOG2E) : 0.f;
        }
        __syncthreads();
        for (int d = tid; d < D; d += nth) {
            float x = 0.f;
#pragma unroll
            for (int r = 0; r < GC; ++r) {
                x += sb[r * D + d];
                sb[r * D + d] = x;
            }
            sc[d] = exp2f(x);
            if (!OUT) sq[d] += x;
        }
        __syncthreads();
        for (int i = tid; i < GC * D; i += nth) {
            const int r = i / D, d = i % D;
            const float x = sb[i];
            if (OUT) sq[r * LQ + d] = bf2f(rq[i]) * p.q_scale * exp2f(x);
            sk[r * LK + d] = bf2f(rk[i]) * exp2f(sb[(GC - 1) * D + d] - x);
        }
        if (OUT) {
            // ---- A: a warp takes whole rows, a long one and a short one in turns
            for (int j = 0; j * nw < GC; ++j) {
                const int r = j * nw + (j & 1 ? nw - 1 - warp : warp);
                if (r >= GC) continue;
                float q[ND], bt[ND];
#pragma unroll
                for (int i = 0; i < ND; ++i) {
                    q[i] = bf2f(rq[r * D + lane + 32 * i]) * p.q_scale;
                    bt[i] = sb[r * D + lane + 32 * i];
                }
                float keep = 0.f;                                    // lane c holds A[r][c]
                for (int c = 0; c <= r; ++c) {
                    float x = 0.f;
#pragma unroll
                    for (int i = 0; i < ND; ++i)
                        x = fmaf(q[i] * bf2f(rk[c * D + lane + 32 * i]), exp2f(bt[i] - sb[c * D + lane + 32 * i]), x);
                    x = warp_sum(x);
                    if (lane == c) keep = x;
                }
                if (lane < GC) sa[r * LA_S + lane] = keep;
            }
        }
        __syncthreads();
        // ---- values of this warp's columns: exact in tf32
        uint32_t v[2][4];
#pragma unroll
        for (int u = 0; u < 2; ++u)
#pragma unroll
            for (int x = 0; x < 4; ++x)
                v[u][x] = __float_as_uint(bf2f(rv[(8 * u + 2 * t + (x >> 1)) * es + warp * 16 + g + 8 * (x & 1)]));
        float o[2][4] = {};
        if (OUT) {
            // ---- O^T [columns][tokens]: from the memory, two groups of eight tokens
            float acc[2][2][4] = {};
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const float4 x0 = *reinterpret_cast<const float4*>(sq + g * LQ + 16 * i + 4 * t);
                const float4 x1 = *reinterpret_cast<const float4*>(sq + (g + 8) * LQ + 16 * i + 4 * t);
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
            // ---- and from the chunk itself
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const float2 x0 = *reinterpret_cast<const float2*>(sa + g * LA_S + 8 * u + 2 * t);
                const float2 x1 = *reinterpret_cast<const float2*>(sa + (g + 8) * LA_S + 8 * u + 2 * t);
                uint32_t h0, l0, h1, l1, h2, l2, h3, l3;
                gl_split(x0.x, h0, l0); gl_split(x0.y, h1, l1); gl_split(x1.x, h2, l2); gl_split(x1.y, h3, l3);
                gl_mma(acc[0][0], v[u], l0, l1);
                gl_mma(acc[1][0], v[u], l2, l3);
                gl_mma(o[0], v[u], h0, h1);
                gl_mma(o[1], v[u], h2, h3);
            }
#pragma unroll
            for (int u = 0; u < 2; ++u)
#pragma unroll
                for (int x = 0; x < 4; ++x) o[u][x] += acc[u][0][x] + acc[u][1][x];
            if (slices == 1) {
                // sums of squares per token over the warp's columns: tokens 8 u + 2 t + (x & 1)
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
            }
        }
        // ---- S <- e^(b_16) S + (k e^(b_16 - b))^T V
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const float4 w = *reinterpret_cast<const float4*>(sc + 16 * i + 4 * t);
            float (&x)[4] = s[2 * i];
            float (&z)[4] = s[2 * i + 1];
            x[0] *= w.x; x[2] *= w.x; x[1] *= w.z; x[3] *= w.z;
            z[0] *= w.y; z[2] *= w.y; z[1] *= w.w; z[3] *= w.w;
        }
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const float* kb = sk + (8 * u + 2 * t) * LK + 2 * g;
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const float2 x0 = *reinterpret_cast<const float2*>(kb + 16 * i), x1 = *reinterpret_cast<const float2*>(kb + LK + 16 * i);
                uint32_t h0, l0, h1, l1, h2, l2, h3, l3;
                gl_split(x0.x, h0, l0); gl_split(x1.x, h1, l1); gl_split(x0.y, h2, l2); gl_split(x1.y, h3, l3);
                gl_mma(s[2 * i], v[u], l0, l1);
                gl_mma(s[2 * i + 1], v[u], l2, l3);
                gl_mma(s[2 * i], v[u], h0, h1);
                gl_mma(s[2 * i + 1], v[u], h2, h3);
            }
        }
        if (OUT) {
            if (slices == 1) {
                // ---- norm and gate, in place of the gate's values; then whole rows go out
                __syncthreads();
#pragma unroll
                for (int u = 0; u < 2; ++u)
#pragma unroll
                    for (int x = 0; x < 2; ++x) {
                        const int r = 8 * u + 2 * t + x;
                        float q2 = 0.f;
                        for (int w = 0; w < nw; ++w) q2 += sn[w * GC + r];
                        const float rs = 1.f / sqrtf(q2 / (float)p.e_n + p.eps);
                        bf16* c = rg + r * es + warp * 16 + g;
                        c[0] = f2bf(o[u][x] * rs * nw0 * gl_silu(bf2f(c[0])));
                        c[8] = f2bf(o[u][x + 2] * rs * nw1 * gl_silu(bf2f(c[8])));
                    }
                __syncthreads();
                for (int i = tid; i < GC * (es / 8); i += nth) {
                    const int r = i / (es / 8), c = (i % (es / 8)) * 8;
                    if (ch * GC + r < n)
                        *reinterpret_cast<uint4*>(reinterpret_cast<bf16*>(p.out) + (tok0 + ch * GC + r) * p.out_s + (long)h * p.E + c) =
                            *reinterpret_cast<const uint4*>(rg + r * es + c);
                }
            } else {
#pragma unroll
                for (int u = 0; u < 2; ++u)
#pragma unroll
                    for (int x = 0; x < 4; ++x) {
                        const int r = 8 * u + 2 * t + (x & 1);
                        if (ch * GC + r < n) p.core[((tok0 + ch * GC + r) * p.H + h) * p.E + e0 + warp * 16 + g + 8 * (x >> 1)] = o[u][x];
                    }
            }
        }
        __syncthreads();                                             // before this stage and the vectors are filled again
    }
    cp_async_wait<0>();
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
        float* w = p.seg_w + (((long)b * p.segs + sgm) * p.H + h) * D;
        for (int d = tid; d < D; d += nth) w[d] = exp2f(sq[d]);
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
    const int cl = a.E <= 32 ? 1 : a.E <= 64 ? 2 : a.E <= 128 ? 4 : 8, cols = (a.E + cl - 1) / cl;
    const size_t fixed = sizeof(float) * (3 * D + 2 * STEP_COLS + 4 + ((a.rank + 3) & ~3)), w2 = (size_t)D * a.rank * (a.w2_f32 ? 4 : 2);
    const int staged = a.rank % 8 == 0 && fixed + w2 <= 48 * 1024;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(a.H * cl, a.B);
    cfg.blockDim = dim3(256);
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
