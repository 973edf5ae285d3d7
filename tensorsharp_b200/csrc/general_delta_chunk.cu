// The generalized delta rule (general_delta.cu) for prompts of bf16 models, eight tokens at a time on the tensor cores.
//
// With c_t the product of the decays w_1 .. w_t of a chunk (per key channel) and, per token,
//   q_t = u_t c_(t-1),   r^_t = r_t c_t,   k^_t = u_t / c_t,   b^_t = a_t u_t / c_t,   v_t (times the key's length)
// the recurrence over the chunk is  p_t = q_t^T S + sum_(s<t) (q_t . k^_s) v_s - (q_t . b^_s) p_s,  so with the 8 x 8 matrices
//   Lk[t][s] = q_t . k^_s,  Lb[t][s] = q_t . b^_s  (s < t),   Mk[t][s] = r^_t . k^_s,  Mb[t][s] = r^_t . b^_s  (s <= t)
//   X = (I + Lb)^-1,   Y = X Lk:      P = X (Q S) + Y V,     O = R S + Mk V - Mb P,     S <- c_8 (S + K^^T V - B^^T P)
// A decay is at least exp(-e^(-1/2)) = 0.545, so 1 / c_t stays below 130 and nothing is lost in f32.
//
//   gdc_prep_kernel   one warp per (chunk, head): the vectors, the 16 x 16 product of (q, r^) with (k^, b^), X and Y
//   gdc_scan_kernel   a warp holds 16 columns and half of the keys of S for the whole prompt, as accumulator fragments of S^T [columns][keys]; an
//                     accumulator tile's two columns per thread are the next product's two k positions (keys are numbered
//                     to suit), so S, Q S and P pass from product to product without leaving the registers
// Products are mma.sync m16n8k8 on tf32 operands split into a high and a low part, three products per term, which keeps
// f32-level accuracy; accumulation, decays and the state are f32.  The norm and gate are gdr_finish_kernel's.
#include "attn_mma.cuh"
#include "common.cuh"
#include "general_delta.cuh"

namespace {
constexpr int CT = 8;                                    // tokens per chunk

// A chunk's record for one head (floats): q and r^ rows | k^ c_8 and -b^ c_8 rows | c_8 | X, Y, Mk, -Mb | values, one
// A fragment per 16 columns.  Row strides keep the fragment loads free of bank conflicts.
template <int D> struct Rec {
    static constexpr int LQ = D + 16, LK = D + 4;
    static constexpr int QR = 0, KB = 16 * LQ, CE = KB + 16 * LK, MX = CE + D, VA = MX + 256, SIZE = VA + 8 * D;
};

// x = hi + lo up to 2^-21 |x|: the tensor core reads the upper 19 bits of an operand
__device__ __forceinline__ void split(float x, uint32_t& hi, uint32_t& lo) {
    hi = __float_as_uint(x) & 0xffffe000u;
    lo = __float_as_uint(x - __uint_as_float(hi));
}
__device__ __forceinline__ void mma_tf32(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
struct Split4 { uint32_t hi[4], lo[4]; };
__device__ __forceinline__ Split4 split4(float a0, float a1, float a2, float a3) {
    Split4 s;
    split(a0, s.hi[0], s.lo[0]); split(a1, s.hi[1], s.lo[1]); split(a2, s.hi[2], s.lo[2]); split(a3, s.hi[3], s.lo[3]);
    return s;
}
// c += A B in f32 accuracy (A split already)
__device__ __forceinline__ void mma3(float (&c)[4], const Split4& a, float b0, float b1) {
    uint32_t h0, l0, h1, l1;
    split(b0, h0, l0);
    split(b1, h1, l1);
    mma_tf32(c, a.lo, h0, h1);
    mma_tf32(c, a.hi, l0, l1);
    mma_tf32(c, a.hi, h0, h1);
}
// first record of sequence b: sequences of any lengths get records of their own
__device__ __forceinline__ long first_record(int q0, int b) { return q0 / CT + b; }
}  // namespace

// ------------------------------------------------------------------------------------------
// Grid (ceil(chunks of the longest sequence * H / 2), B), two warps per CTA, each with its own (chunk, head).
// ------------------------------------------------------------------------------------------
template <int D>
__global__ void __launch_bounds__(64) gdc_prep_kernel(GdrArgs p) {
    using R = Rec<D>;
    constexpr int NV = (D + 127) / 128, LS = D + 4;
    extern __shared__ __align__(16) float sm[];
    const int b = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* rows = sm + warp * (32 * LS + 256);           // [32][LS]: q, r^, k^, b^ of eight tokens each
    float* gram = rows + 32 * LS;                        // [16][16]
    pdl_wait();
    pdl_trigger();
    const int q0 = p.cu_q[b], n = p.cu_q[b + 1] - q0;
    const int id = blockIdx.x * 2 + warp, ch = id / p.H, h = id % p.H;
    if (ch * CT >= n) return;
    const long HD = (long)p.H * D, hc = (long)h * D;
    float* rec = p.pack + ((first_record(q0, b) + ch) * p.H + h) * R::SIZE;
    float c[4 * NV];                                     // the running product of decays
#pragma unroll
    for (int i = 0; i < 4 * NV; ++i) c[i] = 1.f;
#pragma unroll 2
    for (int t = 0; t < CT; ++t) {
        const bool on = ch * CT + t < n;                 // a token past the end changes nothing: w = 1, the rest 0
        const long tok = q0 + ch * CT + (on ? t : 0), row = tok * p.y_s + hc;
        float k[4 * NV], kk = 0.f;
        float4 r4[NV], v4[NV], a4[NV], z4[NV];
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int d = 4 * lane + 128 * i;
            float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
            r4[i] = v4[i] = a4[i] = z4[i] = x;
            if (d < D) {
                x = gd_ld4(p.y, row + HD + d, p.y_f32);
                r4[i] = gd_ld4(p.y, row + d, p.y_f32);
                v4[i] = gd_ld4(p.y, row + 2 * HD + d, p.y_f32);
                a4[i] = gd_ld4(p.y, row + 3 * HD + d, p.y_f32);
                z4[i] = *reinterpret_cast<const float4*>(p.z + tok * p.z_s + hc + d);
            }
            k[4 * i] = x.x; k[4 * i + 1] = x.y; k[4 * i + 2] = x.z; k[4 * i + 3] = x.w;
        }
#pragma unroll
        for (int i = 0; i < 4 * NV; ++i) kk = fmaf(k[i], k[i], kk);
        const float len = sqrtf(warp_sum(kk) + GDR_KEY_EPS), inv = on ? 1.f / len : 0.f, keep = on ? 1.f : 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int d = 4 * lane + 128 * i;
            if (d >= D) continue;
            const float4 ab = *reinterpret_cast<const float4*>(p.ab + hc + d), w0 = *reinterpret_cast<const float4*>(p.w0 + hc + d);
            const float zz[4] = {z4[i].x + w0.x, z4[i].y + w0.y, z4[i].z + w0.z, z4[i].w + w0.w};
            const float aa[4] = {a4[i].x + ab.x, a4[i].y + ab.y, a4[i].z + ab.z, a4[i].w + ab.w};
            const float rr[4] = {r4[i].x, r4[i].y, r4[i].z, r4[i].w}, vv[4] = {v4[i].x, v4[i].y, v4[i].z, v4[i].w};
            float q[4], rh[4], kh[4], bh[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float u = k[4 * i + e] * inv;
                q[e] = u * c[4 * i + e];
                if (on) c[4 * i + e] *= gd_decay(zz[e]);
                const float ic = 1.f / c[4 * i + e];
                rh[e] = keep * rr[e] * c[4 * i + e];
                kh[e] = u * ic;
                bh[e] = gd_sigmoid(aa[e]) * kh[e];
                // value of column d + e as the fragment element of (token t, column): group of 16 columns, lane g * 4 + t / 2
                const int col = d + e, g = col & 7;
                rec[R::VA + (col >> 4) * 128 + (g * 4 + (t >> 1)) * 4 + ((col >> 3) & 1) + 2 * (t & 1)] = keep * vv[e] * len;
            }
            const float4 q4 = make_float4(q[0], q[1], q[2], q[3]), rh4 = make_float4(rh[0], rh[1], rh[2], rh[3]);
            *reinterpret_cast<float4*>(rows + t * LS + d) = q4;
            *reinterpret_cast<float4*>(rows + (8 + t) * LS + d) = rh4;
            *reinterpret_cast<float4*>(rows + (16 + t) * LS + d) = make_float4(kh[0], kh[1], kh[2], kh[3]);
            *reinterpret_cast<float4*>(rows + (24 + t) * LS + d) = make_float4(bh[0], bh[1], bh[2], bh[3]);
            *reinterpret_cast<float4*>(rec + R::QR + t * R::LQ + d) = q4;
            *reinterpret_cast<float4*>(rec + R::QR + (8 + t) * R::LQ + d) = rh4;
        }
    }
    __syncwarp();
    // what survives to the chunk's end
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int d = 4 * lane + 128 * i;
        if (d >= D) continue;
        *reinterpret_cast<float4*>(rec + R::CE + d) = make_float4(c[4 * i], c[4 * i + 1], c[4 * i + 2], c[4 * i + 3]);
#pragma unroll
        for (int t = 0; t < 16; ++t) {
            const float4 x = *reinterpret_cast<const float4*>(rows + (16 + t) * LS + d);
            const float s = t < 8 ? 1.f : -1.f;
            *reinterpret_cast<float4*>(rec + R::KB + t * R::LK + d) =
                make_float4(s * x.x * c[4 * i], s * x.y * c[4 * i + 1], s * x.z * c[4 * i + 2], s * x.w * c[4 * i + 3]);
        }
    }
    // (q, r^) [16 x D] times (k^, b^)^T [D x 16]
    {
        const int g = lane >> 2, t = lane & 3;
        float acc[2][4] = {};
#pragma unroll 4
        for (int k0 = 0; k0 < D; k0 += 8) {
            const float* ap = rows + g * LS + k0 + t;
            const Split4 a = split4(ap[0], ap[8 * LS], ap[4], ap[8 * LS + 4]);
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const float* bp = rows + (16 + 8 * j + g) * LS + k0 + t;
                mma3(acc[j], a, bp[0], bp[4]);
            }
        }
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) gram[(g + 8 * (e >> 1)) * 16 + 8 * j + 2 * t + (e & 1)] = acc[j][e];
    }
    __syncwarp();
    // gram rows 0..7: q, 8..15: r^; columns 0..7: k^, 8..15: b^.  Lane j < 8 solves for column j of X, lane 8 + j for column j of Y
    if (lane < 16) {
        const int j = lane & 7;
        float x[8];
#pragma unroll
        for (int t = 0; t < 8; ++t) {
            float v = lane < 8 ? (t == j ? 1.f : 0.f) : (j < t ? gram[t * 16 + j] : 0.f);
#pragma unroll
            for (int s = 0; s < t; ++s) v = fmaf(-gram[t * 16 + 8 + s], x[s], v);
            x[t] = v;
            rec[R::MX + (lane < 8 ? 0 : 64) + t * 8 + j] = v;
        }
    } else {
        const int j = lane & 7, bcol = lane >= 24 ? 8 : 0;
#pragma unroll
        for (int t = 0; t < 8; ++t) {
            const float v = j <= t ? gram[(8 + t) * 16 + bcol + j] : 0.f;
            rec[R::MX + (bcol ? 192 : 128) + t * 8 + j] = bcol ? -v : v;
        }
    }
}

// ------------------------------------------------------------------------------------------
// Grid (D / 32, H, B), four warps: two groups of 16 columns, each shared by two warps that hold half of the keys.  S^T tile n
// of a warp: rows = columns g, g + 8 of S, tile columns 2 t, 2 t + 1; tile 2 i + e, column m stands for key 16 i + 2 m + e of
// the warp's half.  Consecutive products go to different accumulators, so that none waits for the one before.
// ------------------------------------------------------------------------------------------
template <int D>
__global__ void __launch_bounds__(128) gdc_scan_kernel(GdrArgs p) {
    using R = Rec<D>;
    constexpr int NI = D / 32, VS = 256, BUF = R::VA + VS, ST = 3;
    extern __shared__ __align__(16) float sm[];          // [ST][BUF]: the record up to the values, then this CTA's values; [4][256]
    float* xch = sm + ST * BUF;                          // partial (Q S)^T and (R S)^T of every warp
    const int h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int cg = warp >> 1, half = warp & 1, c0 = blockIdx.x * 32 + cg * 16, k0 = half * (D / 2);
    pdl_wait();
    pdl_trigger();
    const int q0 = p.cu_q[b], n = p.cu_q[b + 1] - q0;
    if (n <= 0) return;
    const int nc = (n + CT - 1) / CT;
    const float* rec = p.pack + (first_record(q0, b) * p.H + h) * R::SIZE;
    const long step = (long)p.H * R::SIZE;
    auto stage = [&](int ch) {                           // every call commits one group, empty past the end
        if (ch < nc) {
            const float* src = rec + ch * step;
            float* dst = sm + (ch % ST) * BUF;
#pragma unroll 4
            for (int i = tid * 4; i < R::VA; i += 512) cp_async16(dst + i, src + i);
            if (tid * 4 < VS) cp_async16(dst + R::VA + tid * 4, src + R::VA + blockIdx.x * VS + tid * 4);
        }
        cp_async_commit();
    };
    stage(0);
    stage(1);
    float* S = p.state + p.seq_slots[b] * p.state_s + (long)h * D * D + (long)c0 * D + k0;
    float s[2 * NI][4];
#pragma unroll
    for (int i = 0; i < NI; ++i)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const float4 x = *reinterpret_cast<const float4*>(S + (g + 8 * r) * D + 16 * i + 4 * t);
            s[2 * i][2 * r] = x.x; s[2 * i + 1][2 * r] = x.y; s[2 * i][2 * r + 1] = x.z; s[2 * i + 1][2 * r + 1] = x.w;
        }
    for (int ch = 0; ch < nc; ++ch) {
        cp_async_wait<1>();
        __syncthreads();                                 // and every warp is done with the chunk whose place is filled next
        stage(ch + 2);
        const float* B = sm + (ch % ST) * BUF;
        // ---- this half's share of (Q S)^T and (R S)^T
        {
            float aq[2][3][4] = {}, ar[2][3][4] = {};
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const float4 bq = *reinterpret_cast<const float4*>(B + R::QR + g * R::LQ + k0 + 16 * i + 4 * t);
                const float4 br = *reinterpret_cast<const float4*>(B + R::QR + (8 + g) * R::LQ + k0 + 16 * i + 4 * t);
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const float (&x)[4] = s[2 * i + e];
                    const Split4 a = split4(x[0], x[2], x[1], x[3]);
                    const Split4 w = split4(e ? bq.y : bq.x, e ? bq.w : bq.z, e ? br.y : br.x, e ? br.w : br.z);
                    mma_tf32(aq[e][0], a.lo, w.hi[0], w.hi[1]);
                    mma_tf32(ar[e][0], a.lo, w.hi[2], w.hi[3]);
                    mma_tf32(aq[e][1], a.hi, w.lo[0], w.lo[1]);
                    mma_tf32(ar[e][1], a.hi, w.lo[2], w.lo[3]);
                    mma_tf32(aq[e][2], a.hi, w.hi[0], w.hi[1]);
                    mma_tf32(ar[e][2], a.hi, w.hi[2], w.hi[3]);
                }
            }
            float q[4], r[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                q[k] = (aq[0][2][k] + aq[1][2][k]) + ((aq[0][0][k] + aq[1][0][k]) + (aq[0][1][k] + aq[1][1][k]));
                r[k] = (ar[0][2][k] + ar[1][2][k]) + ((ar[0][0][k] + ar[1][0][k]) + (ar[0][1][k] + ar[1][1][k]));
            }
            *reinterpret_cast<float4*>(xch + warp * 256 + lane * 4) = make_float4(q[0], q[1], q[2], q[3]);
            *reinterpret_cast<float4*>(xch + warp * 256 + 128 + lane * 4) = make_float4(r[0], r[1], r[2], r[3]);
        }
        // ---- what does not depend on the other half: S <- c_8 S + (K c_8)^T V, and V's part of P
        const float4 v4 = *reinterpret_cast<const float4*>(B + R::VA + cg * 128 + lane * 4);
        const Split4 v = split4(v4.x, v4.y, v4.z, v4.w);
        const float* M = B + R::MX + g * 8 + 2 * t;
        const float2 mx = *reinterpret_cast<const float2*>(M), my = *reinterpret_cast<const float2*>(M + 64);
        const float2 mk = *reinterpret_cast<const float2*>(M + 128), mb = *reinterpret_cast<const float2*>(M + 192);
        const Split4 wm = split4(mx.x, mx.y, my.x, my.y);
        float pa[3][4] = {};
        mma_tf32(pa[0], v.lo, wm.hi[2], wm.hi[3]);
        mma_tf32(pa[1], v.hi, wm.lo[2], wm.lo[3]);
        mma_tf32(pa[2], v.hi, wm.hi[2], wm.hi[3]);
        // one half's rows of K or B (first row of the pair this thread reads) onto all tiles, two i at a time
        auto onto = [&](const Split4& a, const float* kb) {
#pragma unroll
            for (int i = 0; i < NI; i += 2) {
                constexpr int LK = R::LK;
                Split4 w[2];
#pragma unroll
                for (int j = 0; j < 2; ++j)
                    if (i + j < NI) {
                        const float2 x0 = *reinterpret_cast<const float2*>(kb + 16 * (i + j)), x1 = *reinterpret_cast<const float2*>(kb + LK + 16 * (i + j));
                        w[j] = split4(x0.x, x1.x, x0.y, x1.y);
                    }
#pragma unroll
                for (int term = 0; term < 3; ++term)
#pragma unroll
                    for (int j = 0; j < 2; ++j)
                        if (i + j < NI)
#pragma unroll
                            for (int e = 0; e < 2; ++e) {
                                float (&x)[4] = s[2 * (i + j) + e];
                                if (term == 0) mma_tf32(x, a.lo, w[j].hi[2 * e], w[j].hi[2 * e + 1]);
                                else if (term == 1) mma_tf32(x, a.hi, w[j].lo[2 * e], w[j].lo[2 * e + 1]);
                                else mma_tf32(x, a.hi, w[j].hi[2 * e], w[j].hi[2 * e + 1]);
                            }
            }
        };
        const float* kb = B + R::KB + 2 * t * R::LK + k0 + 2 * g;
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const float4 ce = *reinterpret_cast<const float4*>(B + R::CE + k0 + 16 * i + 4 * t);
            float (&x)[4] = s[2 * i];
            float (&y)[4] = s[2 * i + 1];
            x[0] *= ce.x; x[2] *= ce.x; x[1] *= ce.z; x[3] *= ce.z;
            y[0] *= ce.y; y[2] *= ce.y; y[1] *= ce.w; y[3] *= ce.w;
        }
        onto(v, kb);
        __syncthreads();
        // ---- P = X (Q S) + Y V: tile columns 2 t, 2 t + 1 are tokens
        const float4 qa = *reinterpret_cast<const float4*>(xch + (warp & ~1) * 256 + lane * 4);
        const float4 qb = *reinterpret_cast<const float4*>(xch + (warp | 1) * 256 + lane * 4);
        const Split4 q = split4(qa.x + qb.x, qa.z + qb.z, qa.y + qb.y, qa.w + qb.w);
        mma_tf32(pa[0], q.lo, wm.hi[0], wm.hi[1]);
        mma_tf32(pa[1], q.hi, wm.lo[0], wm.lo[1]);
        mma_tf32(pa[2], q.hi, wm.hi[0], wm.hi[1]);
        float pf[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) pf[k] = pa[2][k] + (pa[0][k] + pa[1][k]);
        const Split4 pp = split4(pf[0], pf[2], pf[1], pf[3]);
        // ---- S -= (B c_8)^T P
        onto(pp, kb + 8 * R::LK);
        // ---- O = R S + Mk V - Mb P, eight columns by each half
        {
            const float4 ra = *reinterpret_cast<const float4*>(xch + (warp & ~1) * 256 + 128 + lane * 4);
            const float4 rb = *reinterpret_cast<const float4*>(xch + (warp | 1) * 256 + 128 + lane * 4);
            const Split4 wo = split4(mk.x, mk.y, mb.x, mb.y);
            float oa[3][4] = {};
            mma_tf32(oa[0], v.lo, wo.hi[0], wo.hi[1]);
            mma_tf32(oa[1], v.hi, wo.lo[0], wo.lo[1]);
            mma_tf32(oa[2], v.hi, wo.hi[0], wo.hi[1]);
            mma_tf32(oa[0], pp.lo, wo.hi[2], wo.hi[3]);
            mma_tf32(oa[1], pp.hi, wo.lo[2], wo.lo[3]);
            mma_tf32(oa[2], pp.hi, wo.hi[2], wo.hi[3]);
            const float r[4] = {ra.x + rb.x, ra.y + rb.y, ra.z + rb.z, ra.w + rb.w};
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int tok = ch * CT + 2 * t + e;
                const float o = half ? r[2 + e] + (oa[2][2 + e] + (oa[0][2 + e] + oa[1][2 + e])) : r[e] + (oa[2][e] + (oa[0][e] + oa[1][e]));
                if (tok < n) p.core[((long)(q0 + tok) * p.H + h) * D + c0 + g + 8 * half] = o;
            }
        }
    }
    cp_async_wait<0>();
#pragma unroll
    for (int i = 0; i < NI; ++i)
#pragma unroll
        for (int r = 0; r < 2; ++r)
            *reinterpret_cast<float4*>(S + (g + 8 * r) * D + 16 * i + 4 * t) =
                make_float4(s[2 * i][2 * r], s[2 * i + 1][2 * r], s[2 * i][2 * r + 1], s[2 * i + 1][2 * r + 1]);
}

// ------------------------------------------------------------------------------------------
extern "C" long tsb_general_delta_chunk_floats(int D) { return 41L * D + 576; }        // of a record: Rec<D>::SIZE

template <int D>
static int launch_chunk(const GdrArgs& a, int max_q, cudaStream_t s) {
    static_assert(Rec<D>::SIZE == 41 * D + 576 && Rec<D>::SIZE % 4 == 0 && Rec<D>::VA % 4 == 0, "record");
    const size_t prep = sizeof(float) * 2 * (32 * (D + 4) + 256), scan = sizeof(float) * (3 * (Rec<D>::VA + 256) + 1024);
    static bool configured = false;
    if (!configured) {
        TSB_CHECK_CUDA(cudaFuncSetAttribute(gdc_prep_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)prep));
        TSB_CHECK_CUDA(cudaFuncSetAttribute(gdc_scan_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)scan));
        configured = true;
    }
    const long items = (long)((max_q + CT - 1) / CT) * a.H;
    TSB_CHECK_CUDA(tsb_launch(gdc_prep_kernel<D>, dim3((unsigned)((items + 1) / 2), a.B), dim3(64), prep, s, a));
    // not as a dependent launch: its long-lived CTAs would take the first places that the other kernel's CTAs leave, several
    // on one SM with others idle
    gdc_scan_kernel<D><<<dim3(D / 32, a.H, a.B), 128, scan, s>>>(a);
    return TSB_OK;
}

// Recurrence of a packed batch from prepared projections; pack holds (T / 8 + B + 1) * H records.
extern "C" int tsb_general_delta_chunk(const GdrArgs* args, int max_q, void* stream) {
    const GdrArgs& a = *args;
    int rc = gdr_check(a, "general_delta_chunk");
    if (rc != TSB_OK) return rc;
    TSB_CHECK_ARG(a.z && a.pack && a.core, "general_delta_chunk: missing buffers");
    TSB_CHECK_ARG(a.y_s % 4 == 0 && a.z_s % 4 == 0 && a.out_s % 4 == 0, "general_delta_chunk: rows of %ld / %ld elements", a.y_s, a.z_s);
    if (a.B == 0 || a.T == 0) return TSB_OK;
    cudaStream_t s = (cudaStream_t)stream;
    switch (a.D) {
    case 32: rc = launch_chunk<32>(a, max_q, s); break;
    case 64: rc = launch_chunk<64>(a, max_q, s); break;
    case 96: rc = launch_chunk<96>(a, max_q, s); break;
    case 128: rc = launch_chunk<128>(a, max_q, s); break;
    case 160: rc = launch_chunk<160>(a, max_q, s); break;
    case 192: rc = launch_chunk<192>(a, max_q, s); break;
    case 224: rc = launch_chunk<224>(a, max_q, s); break;
    default: rc = launch_chunk<256>(a, max_q, s); break;
    }
    if (rc != TSB_OK) return rc;
    TSB_CHECK_LAUNCH();
    return tsb_gdr_finish_launch(a, s);
}
