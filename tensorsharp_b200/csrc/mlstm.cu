// mLSTM: a memory per head with exponential gates.  With S [keys, values], a normaliser n [keys] and a running maximum m, per token
//
//   i = cap tanh(zi / cap),  f = log sigmoid(cap tanh(zf / cap)),  m' = max(f + m, i)
//   S <- e^(f + m - m') S + e^(i - m') k v^T,    n <- e^(f + m - m') n + e^(i - m') k
//   o = S^T q / (max(|n . q|, e^-m') + 1e-6),    out = o / rms(o) * norm * sigmoid(g)
//
// Key channels are padded with zeros to D (a multiple of 32) and value channels to E (16, above 128: 32); zero q, k, v keep the
// padding of S zero, and the norm divides by the true size.  The state of a slot is [H][value][key] (S), [H][key] (n), [H] (m).
//
//   steps, 32-bit models   mlstm_step_kernel: token by token; a CTA or a cluster of them per (head, sequence), S in registers;
//                          gates, recurrence, norm and output gate in one kernel
//   prompts, bf16 models   mlstm_gates_kernel finds f, i and m of every token (a scan); mlstm_chunk_kernel takes 64 tokens at a time
//                          on the tensor cores, S in accumulator fragments.  A prompt is cut into segments so that all SMs work: a
//                          first launch finds what every segment adds to an empty memory, mlstm_fold_kernel turns that into
//                          the memory each segment starts from, and a second launch gives the outputs
//
// Within a chunk, with F_t the sum of f up to token t and m0 the maximum ahead of the chunk:
//   num_t = e^(F_t + m0 - m_t) S^T q_t + sum over s <= t of A[t][s] v_s,   A[t][s] = (q_t . k_s) e^(F_t - F_s + i_s - m_t)
//   n . q = e^(F_t + m0 - m_t) n . q_t + sum over s <= t of A[t][s]
//   S <- e^(F_64 + m0 - m_64) S + sum over s of e^(F_64 - F_s + i_s - m_64) k_s v_s^T
// No exponent is positive.  q, k and v are bf16, so q . k is exact in its products; S is read and A multiplied as sums of two bf16 numbers
// (17 bits), what is added to S as a sum of three (24 bits).  Accumulation is f32.
#include <cooperative_groups.h>
#include "attn_mma.cuh"
#include "common.cuh"

namespace cg = cooperative_groups;

struct MlstmArgs {
    const void* y; long y_s; int y_f32;      // projection rows
    long q, k, v, g;                         // first columns of queries, keys (H * D each), values, output gate (H * E each)
    const float* z; long z_s;                // [T, 2 H]: input gates, forget gates
    const float* zb;                         // [2 H]
    const float* norm_w;                     // [H * E]
    float* S; float* n; float* m; long state_s;      // slot stride of all three
    const int* cu_q; const long* seq_slots;
    float* fim;                              // [3][H][T]: f, i and m of every token
    float* m0;                               // [B][H]: m ahead of the batch's tokens
    float* seg;                              // [B][segs][H][E][D]: what a segment adds, then what it starts from (segs > 1)
    float* seg_n;                            // [B][segs][H][D]: the same for n
    float* seg_w;                            // [B][segs][H]: factor of S over a segment
    float* core;                             // [T][H][E] where a head's values are spread over CTAs
    void* out; long out_s; int out_f32;      // [T, H * E]
    int T, B, H, D, E, e_n, segs, seg_len;
    float eps, q_scale, cap;
};

namespace {
constexpr float ML_LOG2E = 1.4426950408889634f;
constexpr float ML_DEN = 1e-6f;
constexpr int ML_MAX_CL = 8;

__device__ __forceinline__ float ml_ld(const void* p, long i, int f32) {
    return f32 ? reinterpret_cast<const float*>(p)[i] : bf2f(reinterpret_cast<const bf16*>(p)[i]);
}
__device__ __forceinline__ float ml_sigmoid(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float ml_exp(float x) {             // x <= 0 up to rounding
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x * ML_LOG2E));
    return r;
}
__device__ __forceinline__ void ml_gates(const MlstmArgs& p, float zi, float zf, int h, float& i, float& f) {
    i = p.cap * tanhf((zi + p.zb[h]) / p.cap);
    const float u = p.cap * tanhf((zf + p.zb[p.H + h]) / p.cap);
    f = fminf(u, 0.f) - log1pf(expf(-fabsf(u)));
}
__device__ __forceinline__ float ml_sum8(float v) {
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    v += __shfl_xor_sync(0xffffffffu, v, 2);
    return v + __shfl_xor_sync(0xffffffffu, v, 4);
}
}  // namespace

// ------------------------------------------------------------------------------------------
// Steps.  Grid (H * CL, B), clusters of CL CTAs along x; a CTA has eight lanes per value column, `cols` columns; D = 8 * KPL.
// ------------------------------------------------------------------------------------------
template <int KPL>
__global__ void __launch_bounds__(KPL <= 16 ? 1024 : 512) mlstm_step_kernel(MlstmArgs p, int cl, int cols) {
    constexpr int D = 8 * KPL, NF = KPL / 4;
    __shared__ __align__(16) float sq[D], sk[D], sn[D];
    __shared__ float sv[128], so[32], sd[32];        // so, sd: per warp, sums of o^2 and of n . q
    __shared__ float ssum[2][ML_MAX_CL];             // every CTA's sum of squares, alternating
    const int h = blockIdx.x / cl, part = blockIdx.x % cl, b = blockIdx.y, tid = threadIdx.x, nt = blockDim.x, l8 = tid & 7, grp = tid >> 3;
    // The state and the batch's metadata are not written by the kernel launched directly before (the projection that makes y), and
    // all kernels before that one have ended: they are on their way while the projection still runs.
    const int q0 = p.cu_q[b], cnt = p.cu_q[b + 1] - q0;
    if (cnt <= 0) return;                                          // the whole cluster
    if (cl > 1) asm volatile("barrier.cluster.arrive.release;" ::: "memory");      // waited for ahead of the first remote store
    const int c0 = part * cols, mine = min(cols, p.E - c0), col = c0 + grp;
    const bool on = grp < mine;
    const long slot = p.seq_slots[b] * p.state_s, hd = (long)h * D;
    float* S = p.S + slot + ((long)h * p.E + (on ? col : 0)) * D + 4 * l8;
    float4 s[NF];
#pragma unroll
    for (int i = 0; i < NF; ++i) s[i] = on ? *reinterpret_cast<const float4*>(S + 32 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
    for (int d = tid; d < D; d += nt) sn[d] = p.n[slot + hd + d];
    float m = p.m[slot + h];
    const float nw = on ? p.norm_w[(long)h * p.E + col] : 0.f;
    pdl_wait();
    pdl_trigger();
    cg::cluster_group cluster = cg::this_cluster();
    if (cl > 1) asm volatile("barrier.cluster.wait.acquire;" ::: "memory");
    for (int t = q0; t < q0 + cnt; ++t) {
        const long row = (long)t * p.y_s;
        for (int d = tid; d < D; d += nt) {
            sq[d] = ml_ld(p.y, row + p.q + hd + d, p.y_f32) * p.q_scale;
            sk[d] = ml_ld(p.y, row + p.k + hd + d, p.y_f32);
        }
        if (tid < mine) sv[tid] = ml_ld(p.y, row + p.v + (long)h * p.E + c0 + tid, p.y_f32);
        const float gate = on && l8 == 0 ? ml_ld(p.y, row + p.g + (long)h * p.E + col, p.y_f32) : 0.f;
        float gi, gf;
        ml_gates(p, p.z[t * p.z_s + h], p.z[t * p.z_s + p.H + h], h, gi, gf);
        const float m1 = fmaxf(gf + m, gi), wa = expf(gf + m - m1), wb = expf(gi - m1);
        m = m1;
        __syncthreads();
        float dot = 0.f;
        for (int d = tid; d < D; d += nt) {                        // every thread its own channels, from token to token
            const float x = fmaf(wa, sn[d], wb * sk[d]);
            sn[d] = x;
            dot = fmaf(x, sq[d], dot);
        }
        const float v = on ? sv[grp] * wb : 0.f;
        float o = 0.f;
#pragma unroll
        for (int i = 0; i < NF; ++i) {
            const int e = 4 * l8 + 32 * i;
            const float4 k = *reinterpret_cast<const float4*>(sk + e), q = *reinterpret_cast<const float4*>(sq + e);
            s[i].x = fmaf(k.x, v, wa * s[i].x); o = fmaf(s[i].x, q.x, o);
            s[i].y = fmaf(k.y, v, wa * s[i].y); o = fmaf(s[i].y, q.y, o);
            s[i].z = fmaf(k.z, v, wa * s[i].z); o = fmaf(s[i].z, q.z, o);
            s[i].w = fmaf(k.w, v, wa * s[i].w); o = fmaf(s[i].w, q.w, o);
        }
        o = on ? ml_sum8(o) : 0.f;
        const float o2 = warp_sum(l8 == 0 ? o * o : 0.f);
        dot = warp_sum(dot);
        if ((tid & 31) == 0) { so[tid >> 5] = o2; sd[tid >> 5] = dot; }
        __syncthreads();
        float ss = 0.f, nq = 0.f;
        for (int w = 0; w < nt >> 5; ++w) nq += sd[w];
        if (cl > 1) {
            // the first warp hands this CTA's sum to every CTA of the cluster: past the barrier each reads its own memory only
            float* sums = ssum[t & 1];
            if (tid < 32) {
                const float x = warp_sum(tid < nt >> 5 ? so[tid] : 0.f);
                if (tid < cl) *cluster.map_shared_rank(sums + part, tid) = x;
            }
            asm volatile("barrier.cluster.arrive.release;" ::: "memory");
            asm volatile("barrier.cluster.wait.acquire;" ::: "memory");
            for (int r = 0; r < cl; ++r) ss += sums[r];
        } else {
            for (int w = 0; w < nt >> 5; ++w) ss += so[w];
        }
        if (t == q0 + cnt - 1) {
            if (on) {
#pragma unroll
                for (int i = 0; i < NF; ++i) *reinterpret_cast<float4*>(S + 32 * i) = s[i];
            }
            if (part == 0) {                                       // (every CTA of the cluster has read them ahead of the barrier)
                for (int d = tid; d < D; d += nt) p.n[slot + hd + d] = sn[d];
                if (tid == 0) p.m[slot + h] = m;
            }
        }
        if (on && l8 == 0) {
            const float den = fmaxf(fabsf(nq), expf(-m)) + ML_DEN;
            const float x = o / den, r = x / sqrtf(ss / den / den / (float)p.e_n + p.eps) * nw * ml_sigmoid(gate);
            const long at = (long)t * p.out_s + (long)h * p.E + col;
            if (p.out_f32) reinterpret_cast<float*>(p.out)[at] = r;
            else reinterpret_cast<bf16*>(p.out)[at] = f2bf(r);
        }
    }
}

// ------------------------------------------------------------------------------------------
// Gates of a prompt: f, i and the running maximum m of every token.  Grid (H, B); a thread has a run of consecutive tokens.  One
// token maps m to max(f + m, i); the map of a run of tokens has the same form, (sum of f, what remains of the i), and the runs are
// composed by a scan over the block.  Also keeps m and n as they were ahead of the batch for the kernels that follow.
// ------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(1024) mlstm_gates_kernel(MlstmArgs p) {
    __shared__ float sf[32], si[32];
    pdl_wait();
    pdl_trigger();
    const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nt = blockDim.x;
    const int q0 = p.cu_q[b], n = p.cu_q[b + 1] - q0;
    if (n <= 0) return;
    const long slot = p.seq_slots[b] * p.state_s;
    if (p.segs == 1)
        for (int d = tid; d < p.D; d += nt) p.seg_n[((long)b * p.H + h) * p.D + d] = p.n[slot + (long)h * p.D + d];
    const int run = (n + nt - 1) / nt, lo = min(n, tid * run), hi = min(n, lo + run);
    float* F = p.fim + (long)h * p.T + q0;
    float* I = F + (long)p.H * p.T;
    float* M = I + (long)p.H * p.T;
    float F0 = 0.f, I0 = -INFINITY;
    constexpr int U = 8;                                           // tokens loaded together; a run of so many stays in registers
    float fr[U], ir[U];
    for (int t0 = lo; t0 < hi; t0 += U) {
        float zi[U], zf[U];
#pragma unroll
        for (int x = 0; x < U; ++x) {
            const float* z = p.z + (long)(q0 + min(t0 + x, hi - 1)) * p.z_s + h;
            zi[x] = z[0];
            zf[x] = z[p.H];
        }
#pragma unroll
        for (int x = 0; x < U; ++x) {
            if (t0 + x >= hi) break;
            float i, f;
            ml_gates(p, zi[x], zf[x], h, i, f);
            F[t0 + x] = fr[x] = f;
            I[t0 + x] = ir[x] = i;
            F0 += f;
            I0 = fmaxf(f + I0, i);
        }
    }
    // inclusive scan over the warp, then over the warps: (a, then b) = (Fa + Fb, max(Fb + Ia, Ib))
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const float pf = __shfl_up_sync(0xffffffffu, F0, o), pi = __shfl_up_sync(0xffffffffu, I0, o);
        if (lane >= o) { I0 = fmaxf(F0 + pi, I0); F0 += pf; }
    }
    if (lane == 31) { sf[warp] = F0; si[warp] = I0; }
    __syncthreads();
    float m = p.m[slot + h];
    if (tid == 0) p.m0[(long)b * p.H + h] = m;
    for (int w = 0; w < warp; ++w) m = fmaxf(sf[w] + m, si[w]);
    const float pf = __shfl_up_sync(0xffffffffu, F0, 1), pi = __shfl_up_sync(0xffffffffu, I0, 1);
    if (lane > 0) m = fmaxf(pf + m, pi);
    if (run <= U) {
#pragma unroll
        for (int x = 0; x < U; ++x)
            if (lo + x < hi) M[lo + x] = m = fmaxf(fr[x] + m, ir[x]);
    } else {
        for (int t = lo; t < hi; ++t) M[t] = m = fmaxf(F[t] + m, I[t]);
    }
    __syncthreads();                                               // everybody has read the slot's m
    if (lo < hi && hi == n) p.m[slot + h] = m;
}

// ------------------------------------------------------------------------------------------
// Prompts.  Grid (segments, H * slices, B); a CTA has a warp per 16 value columns (up to 8), rows of y are bf16.
// S^T of a warp: rows = value columns g, g + 8, tile i's columns = keys 8 i + 2 t, 8 i + 2 t + 1: two neighbouring tiles are an
// operand of the product with the queries.
// ------------------------------------------------------------------------------------------
namespace {
constexpr int MC = 64;                                   // tokens per chunk
constexpr int MLA = MC + 8;                              // row stride of A

// shared memory: two stages of raw rows (q, k, v with padded rows), A as a sum of two, the chunk's vectors
template <int D> struct MlstmShape {
    static constexpr int LD = D + 8;                     // rows of q and k: the eight rows of an ldmatrix start in different banks
    static constexpr int stage(int es, bool out) { return 2 * MC * (LD * (out ? 2 : 1) + es + 8); }
    static constexpr int VECS = 4 * (12 * MC + 8 * MC + D + 16);
    static constexpr int bytes(int es, bool out) { return 2 * stage(es, out) + (out ? 2 * 2 * MC * MLA : 0) + VECS; }
};
__device__ __forceinline__ float2 ml_unpack(uint32_t v) { return __bfloat1622float2(*reinterpret_cast<const bf162*>(&v)); }
// two numbers as sums of N bf16 each
template <int N>
__device__ __forceinline__ void ml_split(float x, float y, uint32_t (&o)[N]) {
#pragma unroll
    for (int i = 0; i < N; ++i) {
        o[i] = pack_bf16(x, y);
        const float2 f = ml_unpack(o[i]);
        x -= f.x;
        y -= f.y;
    }
}
}  // namespace

template <int D, bool OUT>
__global__ void __launch_bounds__(256) mlstm_chunk_kernel(MlstmArgs p, int slices) {
    using Z = MlstmShape<D>;
    constexpr int NI = D / 16, LD = Z::LD;
    extern __shared__ __align__(16) unsigned char raw[];
    const int es = p.E / slices, h = blockIdx.y / slices, e0 = (blockIdx.y % slices) * es, b = blockIdx.z, sgm = blockIdx.x, lv = es + 8;
    const int tid = threadIdx.x, nth = blockDim.x, nw = nth >> 5, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    pdl_wait();
    pdl_trigger();
    const int q0 = p.cu_q[b], n_all = p.cu_q[b + 1] - q0;
    const int from = sgm * p.seg_len, n = min(n_all - from, p.seg_len);
    if (n <= 0 || (!OUT && from + p.seg_len >= n_all)) return;        // (nobody starts from what the last segment leaves)
    const bool last = from + p.seg_len >= n_all;
    const int nc = (n + MC - 1) / MC, stage_bytes = Z::stage(es, OUT);
    const long tok0 = q0 + from;
    bf16* sa = reinterpret_cast<bf16*>(raw + 2 * stage_bytes);       // [2][64][MLA]: A, high and low part
    float* fl = reinterpret_cast<float*>(raw + 2 * stage_bytes + (OUT ? 2 * 2 * MC * MLA : 0));
    float* s_fm = fl;                       // [64] F_t - m_t
    float* s_if = s_fm + MC;                // [64] i_s - F_s
    float* s_m = s_if + MC;                 // [64] m_t
    float* s_in = s_m + MC;                 // [64] e^(F_t + m0 - m_t) q_scale
    float* s_w = s_in + MC;                 // [64] e^(F_64 - F_s + i_s - m_64)
    float* s_qn = s_w + MC;                 // [64] n . q_t
    float* s_den = s_qn + MC;               // [64] 1 / denominator
    float* s_row = s_den + MC;              // [4][64] sums of A over 16 columns
    float* s_misc = s_row + 4 * MC;         // [0] factor of S over the chunk
    float* s_sq = s_misc + MC;              // [8 warps][64] sums of squares
    float* s_n = s_sq + 8 * MC;             // [D]
    const bf16* y = reinterpret_cast<const bf16*>(p.y);

    auto stage = [&](int ch) {
        bf16* dk = reinterpret_cast<bf16*>(raw + (ch & 1) * stage_bytes);
        bf16* dv = dk + MC * LD;
        bf16* dq = dv + MC * lv;
        for (int i = tid; i < MC * (D / 8); i += nth) {
            const int r = i / (D / 8), c = (i % (D / 8)) * 8;
            const bool ok = ch * MC + r < n;
            const long row = (tok0 + ch * MC + (ok ? r : 0)) * p.y_s + (long)h * D + c;
            if (ok) {
                cp_async16(dk + r * LD + c, y + row + p.k);
                if (OUT) cp_async16(dq + r * LD + c, y + row + p.q);
            } else {
                *reinterpret_cast<uint4*>(dk + r * LD + c) = make_uint4(0, 0, 0, 0);
                if (OUT) *reinterpret_cast<uint4*>(dq + r * LD + c) = make_uint4(0, 0, 0, 0);
            }
        }
        for (int i = tid; i < MC * (es / 8); i += nth) {
            const int r = i / (es / 8), c = (i % (es / 8)) * 8;
            if (ch * MC + r < n) cp_async16(dv + r * lv + c, y + (tok0 + ch * MC + r) * p.y_s + (long)h * p.E + e0 + c + p.v);
            else *reinterpret_cast<uint4*>(dv + r * lv + c) = make_uint4(0, 0, 0, 0);
        }
    };
    stage(0);
    cp_async_commit();

    // f, i, m of the first warp's two tokens, one chunk ahead
    const float* fim = p.fim + (long)h * p.T + tok0;
    float f2[2], i2[2], m2[2], m_in = 0.f;
    auto fetch = [&](int ch) {
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const int r = ch * MC + lane + 32 * x;
            const bool ok = r < n;
            f2[x] = ok ? fim[r] : 0.f;
            i2[x] = ok ? fim[(long)p.H * p.T + r] : -1e30f;
            m2[x] = ok ? fim[2L * p.H * p.T + r] : 1e30f;
        }
    };
    if (warp == 0) {
        fetch(0);
        m_in = from > 0 ? fim[2L * p.H * p.T - 1] : p.m0[(long)b * p.H + h];
    }
    const long at_seg = ((long)b * p.segs + sgm) * p.H + h;
    for (int d = tid; d < D; d += nth) s_n[d] = OUT ? p.seg_n[at_seg * D + d] : 0.f;
    float s[2 * NI][4];
    const long head = (long)(e0 + warp * 16) * D;                    // of this warp's columns in a head's state
    const long slot = p.seq_slots[b] * p.state_s;
    float* S_slot = p.S + slot + (long)h * p.E * D + head;
    float* S_seg = p.segs > 1 ? p.seg + at_seg * p.E * D + head : nullptr;
    const float* S0 = S_seg != nullptr ? S_seg : S_slot;
#pragma unroll
    for (int i = 0; i < 2 * NI; ++i)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const float2 x = OUT ? *reinterpret_cast<const float2*>(S0 + (g + 8 * r) * D + 8 * i + 2 * t) : make_float2(0.f, 0.f);
            s[i][2 * r] = x.x;
            s[i][2 * r + 1] = x.y;
        }
    const int ec = warp * 16 + (g & ~1);                             // columns ec, ec + 1, ec + 8, ec + 9 of the results this thread stores
    float2 nw0 = make_float2(0.f, 0.f), nw1 = nw0;
    if (OUT && slices == 1) {
        nw0 = *reinterpret_cast<const float2*>(p.norm_w + (long)h * p.E + ec);
        nw1 = *reinterpret_cast<const float2*>(p.norm_w + (long)h * p.E + ec + 8);
    }
    float total = 1.f;                                               // factor of S over the segment so far (first warp)

    for (int ch = 0; ch < nc; ++ch) {
        cp_async_wait<0>();
        __syncthreads();                                             // this chunk is here, and everybody is done with the one before
        if (ch + 1 < nc) stage(ch + 1);
        cp_async_commit();
        const bf16* rk = reinterpret_cast<const bf16*>(raw + (ch & 1) * stage_bytes);
        const bf16* rv = rk + MC * LD;
        const bf16* rq = rv + MC * lv;
        // ---- the chunk's scalars: a lane has tokens lane and lane + 32
        if (warp == 0) {
            float a = f2[0], c = f2[1];
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float x = __shfl_up_sync(0xffffffffu, a, o), z = __shfl_up_sync(0xffffffffu, c, o);
                if (lane >= o) { a += x; c += z; }
            }
            c += __shfl_sync(0xffffffffu, a, 31);
            const int e = min(MC, n - ch * MC) - 1;                  // the chunk's last token
            const float F_e = __shfl_sync(0xffffffffu, e < 32 ? a : c, e & 31), m_e = __shfl_sync(0xffffffffu, e < 32 ? m2[0] : m2[1], e & 31);
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                const float F = x ? c : a;
                const int r = lane + 32 * x;
                s_fm[r] = F - m2[x];
                s_if[r] = i2[x] - F;
                s_m[r] = m2[x];
                s_in[r] = ml_exp(F + m_in - m2[x]) * p.q_scale;
                s_w[r] = ml_exp(F_e - F + i2[x] - m_e);              // past the end: 0
            }
            const float fac = ml_exp(F_e + m_in - m_e);
            if (lane == 0) s_misc[0] = fac;
            total *= fac;
            m_in = m_e;
            if (ch + 1 < nc) fetch(ch + 1);
        }
        __syncthreads();
        uint32_t gate[8][2];
        if (OUT) {
            if (slices == 1) {
#pragma unroll
                for (int u = 0; u < 8; ++u) {
                    const int r = 8 * u + 2 * t + (g & 1);
                    const bf16* src = y + (tok0 + min(ch * MC + r, n - 1)) * p.y_s + p.g + (long)h * p.E + ec;
                    gate[u][0] = *reinterpret_cast<const uint32_t*>(src);
                    gate[u][1] = *reinterpret_cast<const uint32_t*>(src + 8);
                }
            }
            // ---- A on and below the diagonal, in tiles of 16 x 16
            for (int unit = warp; unit < 10; unit += nw) {
                const int i = unit < 1 ? 0 : unit < 3 ? 1 : unit < 6 ? 2 : 3, j = unit - i * (i + 1) / 2;
                float acc[2][4] = {};
                const bf16* qr = rq + (16 * i + (lane & 15)) * LD + ((lane >> 4) << 3);
                const bf16* kr = rk + (16 * j + ((lane >> 4) << 3) + (lane & 7)) * LD + (((lane >> 3) & 1) << 3);
#pragma unroll 4
                for (int kk = 0; kk < D; kk += 16) {
                    uint32_t qa[4], kb[4];
                    ldsm_x4(qa, qr + kk);
                    ldsm_x4(kb, kr + kk);
                    mma_bf16(acc[0], qa, kb[0], kb[1]);
                    mma_bf16(acc[1], qa, kb[2], kb[3]);
                }
#pragma unroll
                for (int r = 0; r < 2; ++r) {
                    const int tt = 16 * i + g + 8 * r;
                    const float fm = s_fm[tt];
                    float sum = 0.f;
#pragma unroll
                    for (int nt = 0; nt < 2; ++nt) {
                        const int ss = 16 * j + 8 * nt + 2 * t;
                        float a0 = ss <= tt ? acc[nt][2 * r] * p.q_scale * ml_exp(fm + s_if[ss]) : 0.f;
                        float a1 = ss + 1 <= tt ? acc[nt][2 * r + 1] * p.q_scale * ml_exp(fm + s_if[ss + 1]) : 0.f;
                        sum += a0 + a1;
                        uint32_t w[2];
                        ml_split<2>(a0, a1, w);
                        *reinterpret_cast<uint32_t*>(sa + tt * MLA + ss) = w[0];
                        *reinterpret_cast<uint32_t*>(sa + MC * MLA + tt * MLA + ss) = w[1];
                    }
                    sum += __shfl_xor_sync(0xffffffffu, sum, 1);
                    sum += __shfl_xor_sync(0xffffffffu, sum, 2);
                    if (t == 0) s_row[j * MC + tt] = sum;
                }
            }
            // ---- n . q: four lanes per token
            for (int i = tid; i < 4 * MC; i += nth) {
                const bf16* q = rq + (i >> 2) * LD;
                float x = 0.f;
                for (int d = 8 * (i & 3); d < D; d += 32) {
                    const uint4 w = *reinterpret_cast<const uint4*>(q + d);
                    const float4 n0 = *reinterpret_cast<const float4*>(s_n + d), n1 = *reinterpret_cast<const float4*>(s_n + d + 4);
                    const float2 a = ml_unpack(w.x), c = ml_unpack(w.y), e = ml_unpack(w.z), f = ml_unpack(w.w);
                    x = fmaf(a.x, n0.x, x); x = fmaf(a.y, n0.y, x); x = fmaf(c.x, n0.z, x); x = fmaf(c.y, n0.w, x);
                    x = fmaf(e.x, n1.x, x); x = fmaf(e.y, n1.y, x); x = fmaf(f.x, n1.z, x); x = fmaf(f.y, n1.w, x);
                }
                x += __shfl_xor_sync(0xffffffffu, x, 1);
                x += __shfl_xor_sync(0xffffffffu, x, 2);
                if ((i & 3) == 0) s_qn[i >> 2] = x;
            }
            __syncthreads();
            for (int r = tid; r < MC; r += nth) {
                float x = s_in[r] * s_qn[r];
                for (int j = 0; j <= r >> 4; ++j) x += s_row[j * MC + r];
                s_den[r] = 1.f / (fmaxf(fabsf(x), expf(-s_m[r])) + ML_DEN);
            }
        }
        const float fac = s_misc[0];
        for (int d = tid; d < D; d += nth) {                         // n
            float x = fac * s_n[d];
#pragma unroll 8
            for (int r = 0; r < MC; ++r) x = fmaf(s_w[r], bf2f(rk[r * LD + d]), x);
            s_n[d] = x;
        }
        float o[8][4] = {};                                          // [value columns g, g + 8][tokens 8 u + 2 t, + 1]
        if (OUT) {
            const bf16* qr = rq + (((lane >> 4) << 3) + (lane & 7)) * LD + (((lane >> 3) & 1) << 3);
#pragma unroll
            for (int kk = 0; kk < NI; ++kk) {
                uint32_t x0[2], x1[2], x2[2], x3[2];
                ml_split<2>(s[2 * kk][0], s[2 * kk][1], x0);
                ml_split<2>(s[2 * kk][2], s[2 * kk][3], x1);
                ml_split<2>(s[2 * kk + 1][0], s[2 * kk + 1][1], x2);
                ml_split<2>(s[2 * kk + 1][2], s[2 * kk + 1][3], x3);
                const uint32_t hi[4] = {x0[0], x1[0], x2[0], x3[0]}, lo[4] = {x0[1], x1[1], x2[1], x3[1]};
#pragma unroll
                for (int u = 0; u < 4; ++u) {
                    uint32_t qb[4];
                    ldsm_x4(qb, qr + 16 * u * LD + 16 * kk);
                    mma_bf16(o[2 * u], lo, qb[0], qb[1]);
                    mma_bf16(o[2 * u + 1], lo, qb[2], qb[3]);
                    mma_bf16(o[2 * u], hi, qb[0], qb[1]);
                    mma_bf16(o[2 * u + 1], hi, qb[2], qb[3]);
                }
            }
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                const float2 w = *reinterpret_cast<const float2*>(s_in + 8 * u + 2 * t);
                o[u][0] *= w.x; o[u][1] *= w.y; o[u][2] *= w.x; o[u][3] *= w.y;
            }
        }
#pragma unroll
        for (int i = 0; i < 2 * NI; ++i)
#pragma unroll
            for (int x = 0; x < 4; ++x) s[i][x] *= fac;
        // ---- 16 tokens at a time: their values into O^T and into S^T
        const bf16* vr = rv + ((lane & 7) + 8 * (lane >> 4)) * lv + warp * 16 + 8 * ((lane >> 3) & 1);
        const bf16* kr = rk + ((lane & 7) + 8 * ((lane >> 3) & 1)) * LD + 8 * (lane >> 4);
#pragma unroll
        for (int j = 0; j < MC / 16; ++j) {
            uint32_t v[4];
            ldsm_x4_t(v, vr + 16 * j * lv);
            if (OUT) {
                const bf16* ar = sa + (((lane >> 4) << 3) + (lane & 7)) * MLA + 16 * j + (((lane >> 3) & 1) << 3);
#pragma unroll
                for (int u = j; u < 4; ++u)
#pragma unroll
                    for (int x = 1; x >= 0; --x) {
                        uint32_t ab[4];
                        ldsm_x4(ab, ar + x * MC * MLA + 16 * u * MLA);
                        mma_bf16(o[2 * u], v, ab[0], ab[1]);
                        mma_bf16(o[2 * u + 1], v, ab[2], ab[3]);
                    }
            }
            const float2 w0 = *reinterpret_cast<const float2*>(s_w + 16 * j + 2 * t), w1 = *reinterpret_cast<const float2*>(s_w + 16 * j + 8 + 2 * t);
            uint32_t vs[4][3];
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const float2 f = ml_unpack(v[x]), w = x < 2 ? w0 : w1;
                ml_split<3>(f.x * w.x, f.y * w.y, vs[x]);
            }
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                uint32_t kb[4];
                ldsm_x4_t(kb, kr + 16 * j * LD + 16 * i);
#pragma unroll
                for (int x = 2; x >= 0; --x) {
                    const uint32_t va[4] = {vs[0][x], vs[1][x], vs[2][x], vs[3][x]};
                    mma_bf16(s[2 * i], va, kb[0], kb[1]);
                    mma_bf16(s[2 * i + 1], va, kb[2], kb[3]);
                }
            }
        }
        if (!OUT) continue;
        if (slices > 1) {
            __syncthreads();                                         // the denominators
#pragma unroll
            for (int u = 0; u < 8; ++u)
#pragma unroll
                for (int x = 0; x < 4; ++x) {
                    const int r = 8 * u + 2 * t + (x & 1);
                    if (ch * MC + r < n) p.core[((tok0 + ch * MC + r) * p.H + h) * p.E + e0 + warp * 16 + g + 8 * (x >> 1)] = o[u][x] * s_den[r];
                }
            continue;
        }
        // ---- sums of squares per token over the warp's columns
#pragma unroll
        for (int u = 0; u < 8; ++u)
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                float q2 = o[u][x] * o[u][x] + o[u][x + 2] * o[u][x + 2];
                q2 += __shfl_xor_sync(0xffffffffu, q2, 4);
                q2 += __shfl_xor_sync(0xffffffffu, q2, 8);
                q2 += __shfl_xor_sync(0xffffffffu, q2, 16);
                if (g == 0) s_sq[warp * MC + 8 * u + 2 * t + x] = q2;
            }
        __syncthreads();
        // ---- norm and gate: neighbouring lanes trade tokens for columns
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            const int odd = g & 1, r = 8 * u + 2 * t + odd;
            const float y0 = __shfl_xor_sync(0xffffffffu, odd ? o[u][0] : o[u][1], 4), y1 = __shfl_xor_sync(0xffffffffu, odd ? o[u][2] : o[u][3], 4);
            float q2 = 0.f;
            for (int w = 0; w < nw; ++w) q2 += s_sq[w * MC + r];
            if (ch * MC + r >= n) continue;
            const float inv = s_den[r], rs = inv / sqrtf(q2 * inv * inv / (float)p.e_n + p.eps);
            const float2 g0 = ml_unpack(gate[u][0]), g1 = ml_unpack(gate[u][1]);
            const float a0 = odd ? y0 : o[u][0], a1 = odd ? o[u][1] : y0, b0 = odd ? y1 : o[u][2], b1 = odd ? o[u][3] : y1;
            bf16* out = reinterpret_cast<bf16*>(p.out) + (tok0 + ch * MC + r) * p.out_s + (long)h * p.E + ec;
            *reinterpret_cast<uint32_t*>(out) = pack_bf16(a0 * rs * nw0.x * ml_sigmoid(g0.x), a1 * rs * nw0.y * ml_sigmoid(g0.y));
            *reinterpret_cast<uint32_t*>(out + 8) = pack_bf16(b0 * rs * nw1.x * ml_sigmoid(g1.x), b1 * rs * nw1.y * ml_sigmoid(g1.y));
        }
    }
    float* dst = OUT ? (last ? S_slot : nullptr) : S_seg;
    if (dst != nullptr) {
#pragma unroll
        for (int i = 0; i < 2 * NI; ++i)
#pragma unroll
            for (int r = 0; r < 2; ++r)
                *reinterpret_cast<float2*>(dst + (g + 8 * r) * D + 8 * i + 2 * t) = make_float2(s[i][2 * r], s[i][2 * r + 1]);
    }
    float* dn = OUT ? (last ? p.n + slot + (long)h * D : nullptr) : p.seg_n + at_seg * D;
    if (dn != nullptr && e0 == 0) {
        for (int d = tid; d < D; d += nth) dn[d] = s_n[d];           // every thread its own channels
        if (!OUT && tid == 0) p.seg_w[at_seg] = total;
    }
}

// The memory and normaliser every segment starts from: seg[j] <- S, S <- seg_w[j] S + (what segment j adds).  Grid (pieces of
// (E + 1) * D / 4, H, B).
__global__ void __launch_bounds__(256) mlstm_fold_kernel(MlstmArgs p) {
    pdl_wait();
    pdl_trigger();
    const int h = blockIdx.y, b = blockIdx.z, n = p.cu_q[b + 1] - p.cu_q[b];
    const long block = (long)p.E * p.D;
    long i = 4L * (blockIdx.x * 256 + threadIdx.x);
    if (i >= block + p.D || n <= 0) return;
    const bool norm = i >= block;
    if (norm) i -= block;
    const long size = norm ? p.D : block, slot = p.seq_slots[b] * p.state_s + h * size + i;
    const int used = (n + p.seg_len - 1) / p.seg_len;
    float4 s = *reinterpret_cast<const float4*>((norm ? p.n : p.S) + slot);
    for (int j = 0; j < used; ++j) {
        const long at = ((long)b * p.segs + j) * p.H + h;
        float4* c = reinterpret_cast<float4*>((norm ? p.seg_n : p.seg) + at * size + i);
        if (j + 1 == used) {
            *c = s;
            break;
        }
        const float4 x = *c;
        const float w = p.seg_w[at];
        *c = s;
        s = make_float4(fmaf(w, s.x, x.x), fmaf(w, s.y, x.y), fmaf(w, s.z, x.z), fmaf(w, s.w, x.w));
    }
}

// Norm and gate where a head's values are spread over CTAs: one warp per (token, head).
__global__ void __launch_bounds__(256) mlstm_finish_kernel(MlstmArgs p) {
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
        const float r = p.core[id * p.E + e] * rs * p.norm_w[he + e] * ml_sigmoid(ml_ld(p.y, t * p.y_s + p.g + he + e, p.y_f32));
        if (p.out_f32) reinterpret_cast<float*>(p.out)[t * p.out_s + he + e] = r;
        else reinterpret_cast<bf16*>(p.out)[t * p.out_s + he + e] = f2bf(r);
    }
}

// ------------------------------------------------------------------------------------------
static int mlstm_check(const MlstmArgs& a, const char* what) {
    TSB_CHECK_ARG(a.H > 0 && a.D >= 32 && a.D <= 256 && a.D % 32 == 0 && a.E >= 16 && a.E <= 256 && a.E % (a.E > 128 ? 32 : 16) == 0 && a.e_n > 0 && a.e_n <= a.E,
                  "%s: %d heads of %d / %d (true value size %d)", what, a.H, a.D, a.E, a.e_n);
    TSB_CHECK_ARG(a.B <= 65535 && a.H <= 16384 && a.state_s % 4 == 0 && a.cap > 0.f, "%s: %d sequences, %d heads, gates up to %g", what, a.B, a.H, a.cap);
    return TSB_OK;
}

#define MLSTM_SIZES(X) X(32) X(64) X(96) X(128) X(160) X(192) X(224) X(256)

template <int D>
static int launch_mlstm_step(const MlstmArgs& a, cudaStream_t s) {
    // few heads and sequences: their columns spread over the SMs; many: a CTA takes as many as it may
    const int most = D <= 128 ? 128 : 64;
    int cl = (a.E + most - 1) / most;
    while (cl < ML_MAX_CL && a.E > 32 * cl && (long)a.B * a.H * cl < 148) cl *= 2;
    const int cols = (((a.E + cl - 1) / cl) + 3) & ~3;             // whole warps
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(a.H * cl, a.B);
    cfg.blockDim = dim3(8 * cols);
    cfg.stream = s;
    cudaLaunchAttribute at[2];
    at[0].id = cudaLaunchAttributeClusterDimension;
    at[0].val.clusterDim.x = cl;
    at[0].val.clusterDim.y = at[0].val.clusterDim.z = 1;
    at[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = at;
    cfg.numAttrs = tsb_pdl_enabled() ? 2 : 1;
    TSB_CHECK_CUDA(cudaLaunchKernelEx(&cfg, mlstm_step_kernel<D / 8>, a, cl, cols));
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}

extern "C" int tsb_mlstm_step(const MlstmArgs* args, void* stream) {
    const MlstmArgs& a = *args;
    const int rc = mlstm_check(a, "mlstm_step");
    if (rc != TSB_OK) return rc;
    if (a.B == 0) return TSB_OK;
    switch (a.D) {
#define X(D) case D: return launch_mlstm_step<D>(a, (cudaStream_t)stream);
    MLSTM_SIZES(X)
#undef X
    }
    return TSB_ERR_UNSUPPORTED;
}

template <int D>
static int launch_mlstm_prompt(const MlstmArgs& a, int slices, cudaStream_t s) {
    const int es = a.E / slices, threads = 2 * es;                 // a warp per 16 columns
    static bool configured = false;
    if (!configured) {
        TSB_CHECK_CUDA(cudaFuncSetAttribute(mlstm_chunk_kernel<D, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, MlstmShape<D>::bytes(128, false)));
        TSB_CHECK_CUDA(cudaFuncSetAttribute(mlstm_chunk_kernel<D, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, MlstmShape<D>::bytes(128, true)));
        configured = true;
    }
    // the chunk kernels are not dependent launches: their long-lived CTAs would take the first places that the kernel ahead
    // leaves, several on one SM with others idle
    if (a.segs > 1) {
        mlstm_chunk_kernel<D, false><<<dim3(a.segs - 1, a.H * slices, a.B), threads, MlstmShape<D>::bytes(es, false), s>>>(a, slices);
        TSB_CHECK_LAUNCH();
        TSB_CHECK_CUDA(tsb_launch(mlstm_fold_kernel, dim3(((a.E + 1) * a.D / 4 + 255) / 256, a.H, a.B), dim3(256), 0, s, a));
    }
    mlstm_chunk_kernel<D, true><<<dim3(a.segs, a.H * slices, a.B), threads, MlstmShape<D>::bytes(es, true), s>>>(a, slices);
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}

// Recurrence of a packed batch from bf16 projection rows.  `segs` segments of `seg_len` tokens (a multiple of 64) cover the
// longest sequence (max_q tokens); seg and seg_w are needed from two on, core where E is above 128.
extern "C" int tsb_mlstm_prompt(const MlstmArgs* args, int max_q, void* stream) {
    const MlstmArgs& a = *args;
    int rc = mlstm_check(a, "mlstm_prompt");
    if (rc != TSB_OK) return rc;
    const int slices = a.E > 128 ? 2 : 1;
    TSB_CHECK_ARG(!a.y_f32 && !a.out_f32, "mlstm_prompt: bf16 rows and results");
    TSB_CHECK_ARG(((a.y_s | a.q | a.k | a.v | a.g | a.out_s) & 7) == 0, "mlstm_prompt: columns are not 16-byte aligned");
    TSB_CHECK_ARG(a.segs > 0 && a.seg_len > 0 && a.seg_len % MC == 0 && (long)a.segs * a.seg_len >= max_q, "mlstm_prompt: %d segments of %d tokens for %d",
                  a.segs, a.seg_len, max_q);
    TSB_CHECK_ARG(a.fim && a.m0 && a.seg_n && (a.segs == 1 || (a.seg && a.seg_w)) && (slices == 1 || a.core), "mlstm_prompt: missing buffers");
    if (a.B == 0 || a.T == 0) return TSB_OK;
    cudaStream_t s = (cudaStream_t)stream;
    TSB_CHECK_CUDA(tsb_launch(mlstm_gates_kernel, dim3(a.H, a.B), dim3(max_q > 1024 ? 1024 : 256), 0, s, a));
    switch (a.D) {
#define X(D) case D: rc = launch_mlstm_prompt<D>(a, slices, s); break;
    MLSTM_SIZES(X)
#undef X
    }
    if (rc != TSB_OK || slices == 1) return rc;
    TSB_CHECK_CUDA(tsb_launch(mlstm_finish_kernel, dim3((unsigned)(((long)a.T * a.H + 7) / 8)), dim3(256), 0, s, a));
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}
