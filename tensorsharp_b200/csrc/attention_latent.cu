// Latent attention: keys and values of all heads are linear maps of one cached row per token, [latent c (R) | rotated key
// part (rot) | zeros], Lp elements.  Query heads are laid out [dim unrotated | rot rotated | zeros], Dk elements.
//
//   score = (q_c . W_uk c + q_r . k_r) scale = ((W_uk^T q_c) . c + q_r . k_r) scale;   W_uv sum_j p_j c_j = sum_j p_j W_uv c_j
//
// Prompts expand the rows that their queries can see with one matrix product over the cached rows, [W_uk 0; 0 I; W_uv 0],
// and run the ordinary prefill kernel.  Decoding keeps the rows as they are: every query head is mapped into the row's
// space (latent_absorb_kernel), all heads share one row per key, which serves as key and as value
// (latent_decode_kernel, tensor cores), and latent_out_kernel merges the splits with the sink and applies W_uv.
#include "attn_mma.cuh"
#include "common.cuh"

namespace {
__device__ __forceinline__ float la_ld(const void* p, long i, int f32) {
    return f32 ? reinterpret_cast<const float*>(p)[i] : bf2f(reinterpret_cast<const bf16*>(p)[i]);
}
__device__ __forceinline__ void la_st(void* p, long i, int f32, float v) {
    if (f32) reinterpret_cast<float*>(p)[i] = v;
    else reinterpret_cast<bf16*>(p)[i] = f2bf(v);
}
}  // namespace

struct LatentArgs {
    // rows [query latent (qr, padded to qp) | latent (R) | rotated part (rot)]
    const void* y; long y_s; int y_f32;
    const float* qn; const float* kn;        // norm weights [qr], [R]
    const float2* cs;                        // [T, rot / 2]
    const long* slots;                       // [T]
    void* cache;                             // [slots, Lp]
    void* cq;                                // [T, qp]
    int f32;                                 // cache, cq, absorbed queries and results are f32 (else bf16)
    int T, qr, qp, R, rot, Lp;
    float eps;
    // queries
    void* q; int q_f32;                      // [T, H, Dk], not rotated
    const void* wuk; const void* wuv; int w_f32;      // [H * dim, Rp], [H * Dv, Rp]
    void* qa;                                // [T, H, Lp]
    int H, dim, Dk, Rp, Dv;
    // decoding
    const int* block_table; const int* kv_lens;
    float* part_o; float* part_ml;           // [T, H, splits, Ro], [T, H, splits, 2] (null: part_o is the finished result)
    const float* sinks;                      // [H] or null
    void* out;                               // [T, H, Dv]
    float scale;
    int window, page_size, max_pages, splits, Ro;
};

// ------------------------------------------------------------------------------------------
// Norms of both latents, rotation of the shared key part, cache write.  One CTA per token.
// ------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256) latent_prep_kernel(LatentArgs a) {
    __shared__ float red[2][32];
    pdl_wait();
    pdl_trigger();
    const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, w = tid >> 5, nw = blockDim.x >> 5;
    const long row = (long)t * a.y_s, lat = row + a.qp;
    float sq = 0.f, sc = 0.f;
    for (int i = tid; i < a.qr; i += blockDim.x) { const float v = la_ld(a.y, row + i, a.y_f32); sq = fmaf(v, v, sq); }
    for (int i = tid; i < a.R; i += blockDim.x) { const float v = la_ld(a.y, lat + i, a.y_f32); sc = fmaf(v, v, sc); }
    sq = warp_sum(sq);
    sc = warp_sum(sc);
    if (lane == 0) { red[0][w] = sq; red[1][w] = sc; }
    __syncthreads();
    sq = warp_sum(lane < nw ? red[0][lane] : 0.f);
    sc = warp_sum(lane < nw ? red[1][lane] : 0.f);
    const float rq = 1.f / sqrtf(sq / (float)a.qr + a.eps), rc = 1.f / sqrtf(sc / (float)a.R + a.eps);
    for (int i = tid; i < a.qp; i += blockDim.x)
        la_st(a.cq, (long)t * a.qp + i, a.f32, i < a.qr ? la_ld(a.y, row + i, a.y_f32) * rq * a.qn[i] : 0.f);
    const long dst = a.slots[t] * a.Lp;
    const int half = a.rot >> 1;
    for (int i = tid; i < a.Lp; i += blockDim.x) {
        float v = 0.f;
        if (i < a.R) {
            v = la_ld(a.y, lat + i, a.y_f32) * rc * a.kn[i];
        } else if (i < a.R + a.rot) {
            const int e = i - a.R, pair = e < half ? e : e - half;
            const float2 cs = a.cs[(long)t * half + pair];
            const float x0 = la_ld(a.y, lat + a.R + pair, a.y_f32), x1 = la_ld(a.y, lat + a.R + half + pair, a.y_f32);
            v = e < half ? x0 * cs.x - x1 * cs.y : x1 * cs.x + x0 * cs.y;
        }
        la_st(a.cache, dst + i, a.f32, v);
    }
}

extern "C" int tsb_latent_prep(const LatentArgs* args, void* stream) {
    const LatentArgs& a = *args;
    TSB_CHECK_ARG(a.qr > 0 && a.qp >= a.qr && a.R > 0 && a.rot >= 0 && a.rot % 2 == 0 && a.Lp >= a.R + a.rot, "latent_prep: sizes %d / %d / %d in %d",
                  a.qr, a.R, a.rot, a.Lp);
    if (a.T == 0) return TSB_OK;
    TSB_CHECK_CUDA(tsb_launch(latent_prep_kernel, dim3(a.T), dim3(256), 0, (cudaStream_t)stream, a));
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}

// ------------------------------------------------------------------------------------------
// Rotation of the queries' rotated parts in place (prompts).
// ------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256) latent_rotate_kernel(LatentArgs a) {
    pdl_wait();
    pdl_trigger();
    const int half = a.rot >> 1;
    const long i = (long)blockIdx.x * 256 + threadIdx.x;
    if (i >= (long)a.T * a.H * half) return;
    const int pair = (int)(i % half);
    const long th = i / half;
    const float2 cs = a.cs[(th / a.H) * half + pair];
    const long p0 = th * a.Dk + a.dim + pair, p1 = p0 + half;
    const float x0 = la_ld(a.q, p0, a.q_f32), x1 = la_ld(a.q, p1, a.q_f32);
    la_st(a.q, p0, a.q_f32, x0 * cs.x - x1 * cs.y);
    la_st(a.q, p1, a.q_f32, x1 * cs.x + x0 * cs.y);
}

extern "C" int tsb_latent_rotate(const LatentArgs* args, void* stream) {
    const LatentArgs& a = *args;
    TSB_CHECK_ARG(a.rot % 2 == 0 && a.Dk >= a.dim + a.rot, "latent_rotate: head of %d + %d in %d", a.dim, a.rot, a.Dk);
    const long n = (long)a.T * a.H * (a.rot >> 1);
    if (n == 0) return TSB_OK;
    TSB_CHECK_CUDA(tsb_launch(latent_rotate_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, (cudaStream_t)stream, a));
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}

// ------------------------------------------------------------------------------------------
// Queries into the row's space: qa[r] = sum_d W_uk[h, d, r] q[d] for r < R, then the rotated part.  Grid (ceil(Lp / 64), H,
// ceil(T / TT)); eight warps share the d range, a lane holds two neighbouring r.
// ------------------------------------------------------------------------------------------
template <typename TW, int TT>
__global__ void __launch_bounds__(256) latent_absorb_kernel(LatentArgs a) {
    extern __shared__ __align__(16) float sm[];
    float* sq = sm;                          // [Dk][TT]
    float* sp = sm + TT * a.Dk;              // [8][TT][64]
    const int h = blockIdx.y, r0 = blockIdx.x * 64, t0 = blockIdx.z * TT, tid = threadIdx.x, lane = tid & 31, w = tid >> 5;
    const int nt = min(TT, a.T - t0);
    const int r = r0 + 2 * lane;             // Rp is even, columns R .. Rp - 1 are zero
    const TW* wp = reinterpret_cast<const TW*>(a.wuk) + (long)h * a.dim * a.Rp + r;
    float2 wv[8];                            // eight rows of the map in flight per warp, the first ones before the queries are there
    auto fetch = [&](int d0) {
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int d = d0 + 8 * i;
            wv[i] = make_float2(0.f, 0.f);
            if (d < a.dim && r < a.Rp) {
                if (sizeof(TW) == 2) wv[i] = __bfloat1622float2(*reinterpret_cast<const bf162*>(wp + (long)d * a.Rp));
                else wv[i] = *reinterpret_cast<const float2*>(wp + (long)d * a.Rp);
            }
        }
    };
    fetch(w);
    pdl_wait();
    pdl_trigger();
    for (int m = 0; m < TT; ++m)
        for (int d = tid; d < a.Dk; d += 256) sq[d * TT + m] = m < nt ? la_ld(a.q, ((long)(t0 + m) * a.H + h) * a.Dk + d, a.q_f32) : 0.f;
    __syncthreads();
    float acc[TT][2];
#pragma unroll
    for (int m = 0; m < TT; ++m) acc[m][0] = acc[m][1] = 0.f;
    for (int d0 = w; d0 < a.dim; d0 += 64) {
        if (d0 != w) fetch(d0);
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const float* x = sq + min(d0 + 8 * i, a.dim - 1) * TT;
#pragma unroll
            for (int m = 0; m < TT; ++m) {
                acc[m][0] = fmaf(wv[i].x, x[m], acc[m][0]);
                acc[m][1] = fmaf(wv[i].y, x[m], acc[m][1]);
            }
        }
    }
#pragma unroll
    for (int m = 0; m < TT; ++m) *reinterpret_cast<float2*>(sp + (w * TT + m) * 64 + 2 * lane) = make_float2(acc[m][0], acc[m][1]);
    __syncthreads();
    const int half = a.rot >> 1;
    for (int i = tid; i < nt * 64; i += 256) {
        const int m = i / 64, c = i % 64, rr = r0 + c, t = t0 + m;
        if (rr >= a.Lp) continue;
        float v = 0.f;
        if (rr < a.R) {
#pragma unroll
            for (int u = 0; u < 8; ++u) v += sp[(u * TT + m) * 64 + c];
        } else if (rr < a.R + a.rot) {
            const int e = rr - a.R, pair = e < half ? e : e - half;
            const float2 cs = a.cs[(long)t * half + pair];
            const float x0 = sq[(a.dim + pair) * TT + m], x1 = sq[(a.dim + half + pair) * TT + m];
            v = e < half ? x0 * cs.x - x1 * cs.y : x1 * cs.x + x0 * cs.y;
        }
        la_st(a.qa, ((long)t * a.H + h) * a.Lp + rr, a.f32, v);
    }
}

template <typename TW>
static int launch_absorb(const LatentArgs& a, cudaStream_t s) {
    const int bx = (a.Lp + 63) / 64;
    // tokens per CTA: each shares the head's weights between its tokens; few tokens keep one for parallelism
    if (a.T <= 2) {
        const size_t smem = sizeof(float) * (a.Dk + 8 * 64);
        TSB_CHECK_CUDA(tsb_launch(latent_absorb_kernel<TW, 1>, dim3(bx, a.H, a.T), dim3(256), smem, s, a));
    } else {
        const size_t smem = sizeof(float) * 4 * (a.Dk + 8 * 64);
        TSB_CHECK_CUDA(tsb_launch(latent_absorb_kernel<TW, 4>, dim3(bx, a.H, (a.T + 3) / 4), dim3(256), smem, s, a));
    }
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}

extern "C" int tsb_latent_absorb(const LatentArgs* args, void* stream) {
    const LatentArgs& a = *args;
    TSB_CHECK_ARG(a.Rp % 2 == 0 && a.Rp >= a.R && a.Lp >= a.R + a.rot && a.Dk >= a.dim + a.rot && a.Dk <= 1024 && a.H <= 65535 && a.T <= 4 * 65535,
                  "latent_absorb: latent %d (%d), head %d + %d in %d", a.R, a.Rp, a.dim, a.rot, a.Dk);
    if (a.T == 0) return TSB_OK;
    return a.w_f32 ? launch_absorb<float>(a, (cudaStream_t)stream) : launch_absorb<bf16>(a, (cudaStream_t)stream);
}

// ------------------------------------------------------------------------------------------
// Decode attention over the cached rows.  Grid (splits, ceil(H / (16 MT)), B), eight warps; 16 MT query heads are the rows of
// MT m16 tiles.  Rows of the cache arrive in tiles of 64 keys through cp.async, two stages.  For the scores a warp takes half
// of the keys and a quarter of the row's columns, for which it keeps the queries in registers (QS k-steps of 16 at most), so a
// tile's keys are read from shared memory once; the quarters are added where the softmax is taken.  For the values warp w
// accumulates the latent columns 16 (w NV + i).
// ------------------------------------------------------------------------------------------
template <int NV, int QS, int MT>
__global__ void __launch_bounds__(256) latent_decode_kernel(LatentArgs a) {
    constexpr int KT = 64, LDP = KT + 8, LDS_ = KT + 8, ROWS = 16 * MT, TPR = 256 / ROWS, KPT = KT / TPR;      // threads per row, keys each
    constexpr float LOG2E = 1.4426950408889634f;
    extern __shared__ __align__(128) unsigned char smem_raw[];
    __shared__ float scorr[ROWS];
    const int ld = a.Lp + 8, cl = a.Lp / 8;
    bf16* sK = reinterpret_cast<bf16*>(smem_raw);       // [2][64][ld]
    bf16* sP = sK + 2 * KT * ld;                        // [ROWS][LDP]
    bf16* sQ = sP + ROWS * LDP;                         // [ROWS][ld], later:
    float* sS = reinterpret_cast<float*>(sQ);           // [4][ROWS][LDS_] scores by quarters
    const int split = blockIdx.x, h0 = blockIdx.y * ROWS, b = blockIdx.z, G = min(ROWS, a.H - h0);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, kq = warp & 3, kg = warp >> 2;
    // The cached rows and the batch's metadata are not written by the kernel launched directly before (the one that makes
    // qa), and all kernels before that one have ended: the first tile is on its way before the queries are there.
    const int len = a.kv_lens[b];
    const int lo = (a.window > 0 && len > a.window) ? len - a.window : 0;
    const int per = (((len - lo + a.splits - 1) / a.splits) + 31) & ~31;
    const int s0 = lo + split * per, s1 = min(len, s0 + per);
    const bf16* cache = reinterpret_cast<const bf16*>(a.cache);
    auto load_tile = [&](int base, int stage) {
        const int r = tid >> 2, j = base + r;           // four threads per row
        bf16* dst = sK + (stage * KT + r) * ld;
        if (j < s1) {
            const long slot = (long)a.block_table[(long)b * a.max_pages + j / a.page_size] * a.page_size + j % a.page_size;
            for (int c = tid & 3; c < cl; c += 4) cp_async16(dst + c * 8, cache + slot * a.Lp + c * 8);
        } else {
            for (int c = tid & 3; c < cl; c += 4) *reinterpret_cast<uint4*>(dst + c * 8) = make_uint4(0u, 0u, 0u, 0u);
        }
        cp_async_commit();
    };
    const int steps = a.Lp / 16, qs = (steps + 3) / 4, k_lo = kq * qs, k_n = max(0, min(qs, steps - k_lo));      // k-steps of this warp
    uint32_t qf[MT][QS][4];
    if (s0 < s1) load_tile(s0, 0);
    pdl_wait();
    pdl_trigger();
    if (s0 < s1) {
        for (int i = tid; i < ROWS * cl; i += 256) {
            const int r = i / cl, c = i - r * cl;
            uint4 v = make_uint4(0u, 0u, 0u, 0u);
            if (r < G) v = *reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(a.qa) + ((long)b * a.H + h0 + r) * a.Lp + c * 8);
            *reinterpret_cast<uint4*>(sQ + r * ld + c * 8) = v;
        }
        __syncthreads();
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int i = 0; i < QS; ++i)
                if (i < k_n) ldsm_x4(qf[m][i], sQ + (16 * m + (lane & 15)) * ld + (k_lo + i) * 16 + ((lane >> 4) << 3));
        __syncthreads();                                 // the queries' place is the scores' from here on
    }
    float o[MT][2 * NV][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int i = 0; i < 2 * NV; ++i) o[m][i][0] = o[m][i][1] = o[m][i][2] = o[m][i][3] = 0.f;
    const int row = tid / TPR, key0 = (tid % TPR) * KPT;             // this thread's part of the softmax
    float mrow = -INFINITY, lrow = 0.f;
    int stage = 0;
    for (int base = s0; base < s1; base += KT, stage ^= 1) {
        cp_async_wait<0>();
        __syncthreads();                                 // the tile is there, and the last one is done with
        if (base + KT < s1) load_tile(base + KT, stage ^ 1);
        const bf16* tK = sK + stage * KT * ld;
        {
            float s[MT][4][4];
#pragma unroll
            for (int m = 0; m < MT; ++m)
#pragma unroll
                for (int i = 0; i < 4; ++i) s[m][i][0] = s[m][i][1] = s[m][i][2] = s[m][i][3] = 0.f;
            const bf16* krow = tK + (kg * 32 + ((lane >> 4) << 3) + (lane & 7)) * ld + k_lo * 16 + (((lane >> 3) & 1) << 3);
#pragma unroll
            for (int i = 0; i < QS; ++i) {
                if (i >= k_n) break;
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    uint32_t kb[4];
                    ldsm_x4(kb, krow + half * 16 * ld + i * 16);
#pragma unroll
                    for (int m = 0; m < MT; ++m) {
                        mma_bf16(s[m][2 * half], qf[m][i], kb[0], kb[1]);
                        mma_bf16(s[m][2 * half + 1], qf[m][i], kb[2], kb[3]);
                    }
                }
            }
#pragma unroll
            for (int m = 0; m < MT; ++m)
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int r = 0; r < 2; ++r)
                        *reinterpret_cast<float2*>(sS + (kq * ROWS + 16 * m + (lane >> 2) + 8 * r) * LDS_ + kg * 32 + i * 8 + (lane & 3) * 2) =
                            make_float2(s[m][i][2 * r], s[m][i][2 * r + 1]);
        }
        __syncthreads();
        {
            float p[KPT], m = mrow;
#pragma unroll
            for (int j = 0; j < KPT; j += 4) {
                float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                for (int q = 0; q < 4; ++q) {
                    const float4 x = *reinterpret_cast<const float4*>(sS + (q * ROWS + row) * LDS_ + key0 + j);
                    v.x += x.x; v.y += x.y; v.z += x.z; v.w += x.w;
                }
                p[j] = v.x; p[j + 1] = v.y; p[j + 2] = v.z; p[j + 3] = v.w;
            }
#pragma unroll
            for (int j = 0; j < KPT; ++j) {
                p[j] = base + key0 + j < s1 ? p[j] * a.scale : -INFINITY;
                m = fmaxf(m, p[j]);
            }
#pragma unroll
            for (int x = TPR / 2; x >= 1; x >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, x));      // the tile has a valid key: finite
            const float corr = mrow == -INFINITY ? 0.f : exp2f((mrow - m) * LOG2E);
            mrow = m;
            lrow *= corr;
#pragma unroll
            for (int j = 0; j < KPT; j += 2) {
                const float e0 = exp2f((p[j] - m) * LOG2E), e1 = exp2f((p[j + 1] - m) * LOG2E);
                lrow += e0 + e1;
                *reinterpret_cast<uint32_t*>(sP + row * LDP + key0 + j) = pack_bf16(e0, e1);
            }
            if (tid % TPR == 0) scorr[row] = corr;
        }
        __syncthreads();
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            const float c0 = scorr[16 * m + (lane >> 2)], c1 = scorr[16 * m + (lane >> 2) + 8];
#pragma unroll
            for (int i = 0; i < 2 * NV; ++i) {
                o[m][i][0] *= c0; o[m][i][1] *= c0;
                o[m][i][2] *= c1; o[m][i][3] *= c1;
            }
        }
#pragma unroll
        for (int kt = 0; kt < KT / 16; ++kt) {
            uint32_t pa[MT][4];
#pragma unroll
            for (int m = 0; m < MT; ++m) ldsm_x4(pa[m], sP + (16 * m + (lane & 15)) * LDP + kt * 16 + ((lane >> 4) << 3));
            const bf16* vrow = tK + (kt * 16 + (((lane >> 3) & 1) << 3) + (lane & 7)) * ld + ((lane >> 4) << 3);
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const int c = (warp * NV + i) * 16;
                if (c >= a.R) break;
                uint32_t vb[4];
                ldsm_x4_t(vb, vrow + c);
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    mma_bf16(o[m][2 * i], pa[m], vb[0], vb[1]);
                    mma_bf16(o[m][2 * i + 1], pa[m], vb[2], vb[3]);
                }
            }
        }
    }
#pragma unroll
    for (int x = TPR / 2; x >= 1; x >>= 1) lrow += __shfl_xor_sync(0xffffffffu, lrow, x);
    const long p0 = ((long)b * a.H + h0) * a.splits + split;             // partial of head h0 + r: p0 + r * splits
    if (row < G && tid % TPR == 0) {
        a.part_ml[(p0 + (long)row * a.splits) * 2] = mrow;
        a.part_ml[(p0 + (long)row * a.splits) * 2 + 1] = lrow;
    }
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int hr = 16 * m + (lane >> 2) + 8 * r;
            if (hr >= G) continue;
#pragma unroll
            for (int i = 0; i < 2 * NV; ++i) {
                const int c = (warp * NV + (i >> 1)) * 16 + (i & 1) * 8 + (lane & 3) * 2;
                if (c < a.Ro) *reinterpret_cast<float2*>(a.part_o + (p0 + (long)hr * a.splits) * a.Ro + c) = make_float2(o[m][i][2 * r], o[m][i][2 * r + 1]);
            }
        }
}

static size_t latent_decode_smem(int Lp, int MT) {
    const size_t ld = Lp + 8, q = 16 * MT * ld * sizeof(bf16), sc = (size_t)4 * 16 * MT * 72 * sizeof(float);
    return (2 * 64 * ld + 16 * MT * 72) * sizeof(bf16) + (q > sc ? q : sc);
}

template <int NV, int QS, int MT>
static int launch_latent_decode(const LatentArgs& a, cudaStream_t s) {
    const size_t smem = latent_decode_smem(a.Lp, MT);
    static size_t configured = 0;
    if (smem > configured) {
        TSB_CHECK_CUDA(cudaFuncSetAttribute(latent_decode_kernel<NV, QS, MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        configured = smem;
    }
    TSB_CHECK_CUDA(tsb_launch(latent_decode_kernel<NV, QS, MT>, dim3(a.splits, (a.H + 16 * MT - 1) / (16 * MT), a.T), dim3(256), smem, s, a));
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}

// Tiles of 16 query heads per CTA of the decode kernel: two where there are more than 16 heads, sequences enough to fill the
// SMs all the same, and room
static int latent_head_tiles(int B, int H, int Lp) { return H > 16 && B >= 4 && latent_decode_smem(Lp, 2) <= 226 * 1024 ? 2 : 1; }
extern "C" int tsb_latent_heads_per_cta(int B, int H, int Lp) { return 16 * latent_head_tiles(B, H, Lp); }
extern "C" long tsb_latent_decode_smem(int B, int H, int Lp) { return (long)latent_decode_smem(Lp, latent_head_tiles(B, H, Lp)); }

template <int NV, int QS>
static int launch_latent_decode_mt(const LatentArgs& a, cudaStream_t s) {
    // rows with a wide rotated part need more k-steps than the latent size suggests
    const bool two = latent_head_tiles(a.T, a.H, a.Lp) == 2;
    if (a.Lp > 64 * QS) return two ? launch_latent_decode<NV, 11, 2>(a, s) : launch_latent_decode<NV, 11, 1>(a, s);
    return two ? launch_latent_decode<NV, QS, 2>(a, s) : launch_latent_decode<NV, QS, 1>(a, s);
}

// One query per sequence (T sequences); leaves the split partials in part_o / part_ml.
extern "C" int tsb_latent_decode(const LatentArgs* args, void* stream) {
    const LatentArgs& a = *args;
    TSB_CHECK_ARG(!a.f32 && a.Lp % 32 == 0 && a.Lp <= 704 && a.R > 0 && a.R <= 512 && a.Lp >= a.R + a.rot, "latent_decode: latent %d + %d in %d (limits 512, 704)",
                  a.R, a.rot, a.Lp);
    TSB_CHECK_ARG(a.splits >= 1 && a.splits <= 64 && a.part_o && a.part_ml && a.Ro % 8 == 0 && a.Ro >= a.R && a.Ro <= ((a.R + 15) & ~15),
                  "latent_decode: %d splits, partial rows of %d", a.splits, a.Ro);
    if (a.T == 0) return TSB_OK;
    cudaStream_t s = (cudaStream_t)stream;
    switch ((a.R + 127) / 128) {
    case 1: return launch_latent_decode_mt<1, 3>(a, s);
    case 2: return launch_latent_decode_mt<2, 5>(a, s);
    case 3: return launch_latent_decode_mt<3, 7>(a, s);
    default: return launch_latent_decode_mt<4, 9>(a, s);
    }
}

// ------------------------------------------------------------------------------------------
// Merge of the splits (with the sink) and the value map.  A cluster of CTAs per (head, token), eight warps each: every CTA
// merges a share of the latent columns, hands them to the others through distributed shared memory, and then computes a
// share of the output rows, one row of W_uv per warp at a time.
// ------------------------------------------------------------------------------------------
// *p of CTA `rank` of the cluster = v
__device__ __forceinline__ void cluster_store(float* p, int rank, float v) {
    uint32_t a;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(a) : "r"((uint32_t)__cvta_generic_to_shared(p)), "r"(rank));
    asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(a), "f"(v) : "memory");
}
__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }

template <typename TW>
__device__ __forceinline__ void la_row8(const TW* p, float (&v)[8]) {
    if (sizeof(TW) == 2) {
        const uint4 r = *reinterpret_cast<const uint4*>(p);
        const uint32_t* x = reinterpret_cast<const uint32_t*>(&r);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            v[2 * c] = __uint_as_float(x[c] << 16);
            v[2 * c + 1] = __uint_as_float(x[c] & 0xffff0000u);
        }
    } else {
#pragma unroll
        for (int c = 0; c < 8; ++c) v[c] = (float)p[c];
    }
}

template <typename TW>
__global__ void __launch_bounds__(256) latent_out_kernel(LatentArgs a, int rows) {
    extern __shared__ __align__(16) float sm[];          // [Rp]
    __shared__ float cw[64], share[256];
    const int cs = gridDim.x, rank = blockIdx.x;         // the cluster spans the grid's x
    const int e0 = rank * rows, e1 = min(a.Dv, e0 + rows), h = blockIdx.y, t = blockIdx.z;
    const int tid = threadIdx.x, lane = tid & 31, w = tid >> 5;
    if (cs > 1) cluster_arrive();
    const TW* wuv = reinterpret_cast<const TW*>(a.wuv) + (long)h * a.Dv * a.Rp;
    float first[2][8];                                   // this warp's first row, up to 512 columns of it
#pragma unroll
    for (int i = 0; i < 2; ++i)
        if (e0 + w < e1 && lane * 8 + 256 * i < a.Rp) la_row8(wuv + (long)(e0 + w) * a.Rp + lane * 8 + 256 * i, first[i]);
    pdl_wait();
    pdl_trigger();
    const long th = (long)t * a.H + h;
    if (a.part_ml == nullptr) {
        for (int r = tid; r < a.Rp; r += 256) sm[r] = r < a.R ? a.part_o[th * a.Ro + r] : 0.f;
    } else {
        const float* ml = a.part_ml + th * a.splits * 2;
        if (w == 0) {                                    // the splits' weights, at most 64
            const float s0 = a.sinks ? a.sinks[h] : -INFINITY;
            const float m0 = lane < a.splits ? ml[2 * lane] : -INFINITY, m1 = lane + 32 < a.splits ? ml[2 * lane + 64] : -INFINITY;
            const float l0 = lane < a.splits ? ml[2 * lane + 1] : 0.f, l1 = lane + 32 < a.splits ? ml[2 * lane + 65] : 0.f;
            const float m = fmaxf(s0, warp_max(fmaxf(m0, m1)));
            const float c0 = m0 == -INFINITY ? 0.f : expf(m0 - m), c1 = m1 == -INFINITY ? 0.f : expf(m1 - m);
            const float inv = 1.f / (warp_sum(l0 * c0 + l1 * c1) + (a.sinks ? expf(s0 - m) : 0.f));
            cw[lane] = c0 * inv;
            cw[lane + 32] = c1 * inv;
        }
        __syncthreads();
        if (cs > 1) cluster_wait();                      // the other CTAs have started: their memory may be written
        // this CTA's columns [c0, c1): G groups of threads share the splits of a column
        const float* po = a.part_o + th * a.splits * a.Ro;
        const int per = (((a.Rp + cs - 1) / cs) + 63) & ~63, c0 = min(a.Rp, rank * per), c1 = min(a.Rp, c0 + per);
        const int G = per == 64 ? 4 : per == 128 ? 2 : 1, lanes = 256 / G, grp = tid / lanes;
        for (int r = c0 + tid % lanes; r < c0 + per; r += lanes) {        // with G > 1 one turn for every thread
            float v = 0.f;
            if (r < a.R && r < c1) {
#pragma unroll 8
                for (int i = grp; i < a.splits; i += G) v = fmaf(po[(long)i * a.Ro + r], cw[i], v);      // an empty split holds zeros
            }
            if (G > 1) {
                share[tid] = v;
                __syncthreads();
                if (grp == 0)
                    for (int i = 1; i < G; ++i) v += share[tid + i * lanes];
            }
            if (grp == 0 && r < c1)
                for (int c = 0; c < cs; ++c) cluster_store(sm + r, c, v);
        }
    }
    if (cs > 1) {
        cluster_arrive();
        cluster_wait();
    }
    __syncthreads();
    auto dot8 = [&](const float (&v)[8], int u, float acc) {
        const float4 x0 = *reinterpret_cast<const float4*>(sm + u), x1 = *reinterpret_cast<const float4*>(sm + u + 4);
        acc = fmaf(v[0], x0.x, acc); acc = fmaf(v[1], x0.y, acc); acc = fmaf(v[2], x0.z, acc); acc = fmaf(v[3], x0.w, acc);
        acc = fmaf(v[4], x1.x, acc); acc = fmaf(v[5], x1.y, acc); acc = fmaf(v[6], x1.z, acc); return fmaf(v[7], x1.w, acc);
    };
    if (e0 + w < e1) {
        float acc = 0.f;
#pragma unroll
        for (int i = 0; i < 2; ++i)
            if (lane * 8 + 256 * i < a.Rp) acc = dot8(first[i], lane * 8 + 256 * i, acc);
        for (int u = lane * 8 + 512; u < a.Rp; u += 256) {
            float v[8];
            la_row8(wuv + (long)(e0 + w) * a.Rp + u, v);
            acc = dot8(v, u, acc);
        }
        acc = warp_sum(acc);
        if (lane == 0) la_st(a.out, th * a.Dv + e0 + w, a.f32, acc);
    }
    for (int e = e0 + w + 8; e < e1; e += 32) {          // the others, four at a time
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
        for (int u = lane * 8; u < a.Rp; u += 256) {     // Rp is a multiple of 8
            float v[4][8];
#pragma unroll
            for (int j = 0; j < 4; ++j) la_row8(wuv + (long)min(e + 8 * j, e1 - 1) * a.Rp + u, v[j]);
#pragma unroll
            for (int j = 0; j < 4; ++j) acc[j] = dot8(v[j], u, acc[j]);
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            acc[j] = warp_sum(acc[j]);
            if (lane == 0 && e + 8 * j < e1) la_st(a.out, th * a.Dv + e + 8 * j, a.f32, acc[j]);
        }
    }
}

extern "C" int tsb_latent_out(const LatentArgs* args, void* stream) {
    const LatentArgs& a = *args;
    TSB_CHECK_ARG(a.Rp % 8 == 0 && a.Rp >= a.R && a.Rp <= 4096 && a.Dv > 0 && a.T <= 65535 && a.H <= 65535, "latent_out: latent %d (%d), values %d, %d rows",
                  a.R, a.Rp, a.Dv, a.T);
    if (a.T == 0) return TSB_OK;
    // CTAs per (head, token): as many as keep all of them on the SMs together
    int cs = 1;
    while (cs < 8 && a.part_ml != nullptr && (long)a.T * a.H * cs * 2 <= 1184) cs *= 2;
    const int rows = (((a.Dv + cs - 1) / cs) + 7) & ~7;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(cs, a.H, a.T);
    cfg.blockDim = dim3(256);
    cfg.dynamicSmemBytes = sizeof(float) * a.Rp;
    cfg.stream = (cudaStream_t)stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = cs;
    attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = tsb_pdl_enabled() ? 2 : 1;
    if (a.w_f32) TSB_CHECK_CUDA(cudaLaunchKernelEx(&cfg, latent_out_kernel<float>, a, rows));
    else TSB_CHECK_CUDA(cudaLaunchKernelEx(&cfg, latent_out_kernel<bf16>, a, rows));
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}
