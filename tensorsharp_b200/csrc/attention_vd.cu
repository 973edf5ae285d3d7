// Attention over the paged bf16 cache for key and value head sizes of their own: q, k [.., Dh], v, out [.., Dv], both
// multiples of 16 up to 256 (the kernels of attention.cu keep the sizes 64 / 128 / 256 / 512 with Dv = Dh).
//
// Same structure as those kernels: flash prefill on mma.sync m16n8k16 (64 queries x one head per CTA, 64-key tiles through
// cp.async, two stages), and split-KV decode with the query heads of a KV head as the rows of one m16 tile, merged by
// attn_combine_kernel.  Two differences follow from the sizes: the key size is a run-time loop bound (Q fragments are read
// from shared memory where they are used; only the accumulators, whose number depends on Dv, are registers), and tile rows
// are padded by 16 bytes instead of XOR-swizzled: with an even number of 16-byte pieces per row the padded row length is
// odd in units of 16 bytes, so the eight rows of an ldmatrix start in eight different bank groups.
//
// These kernels also know a window with kept first positions (two ranges of key tiles), a distance bias per head, a gate per
// output column, and caches whose rows are key and value at once (AttnArgs::kv_scale): one tile is then staged and read both
// ways, and the scores get the factor of their key.  They are instances of their own (FORM 1), which leaves the others as they are.
// Further instances (FORM 2) know all of that, a distance bias r1 ln(1 + r2 d), and weights sigmoid(score + bias) in place of the
// softmax: those need no running maximum and no sum.  In prompts the bias of a tile's 127 distances is found once, by one thread each.
#include "attn_args.cuh"
#include "attn_mma.cuh"
#include "common.cuh"

__device__ __forceinline__ long vd_slot(const AttnArgs& a, int b, int j) {
    return (long)a.block_table[(long)b * a.max_pages + j / a.page_size] * a.page_size + j % a.page_size;
}

// The accumulator tile of one 64- or 32-key step: online softmax of the 16 x KT scores `s` of a warp (row r of the thread:
// lane / 4 + 8 r), masked by the caller; P V is left to the caller.  Scores are unscaled; f = scale.
template <int KT, int NO>
__device__ __forceinline__ void vd_softmax(float (&s)[KT / 8][4], float (&o)[NO][4], float (&mrow)[2], float (&lrow)[2], float f) {
    constexpr float LOG2E = 1.4426950408889634f;
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int nt = 0; nt < KT / 8; ++nt) {
        mx[0] = fmaxf(mx[0], fmaxf(s[nt][0], s[nt][1]));
        mx[1] = fmaxf(mx[1], fmaxf(s[nt][2], s[nt][3]));
    }
    float corr[2], mneg[2], rsum[2] = {0.f, 0.f};
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
        mx[r] = fmaxf(mrow[r], mx[r] * f);
        corr[r] = (mrow[r] == -INFINITY) ? 0.f : exp2f((mrow[r] - mx[r]) * LOG2E);
        mrow[r] = mx[r];
        mneg[r] = (mx[r] == -INFINITY) ? 0.f : -mx[r] * LOG2E;
    }
    const float fl = f * LOG2E;
#pragma unroll
    for (int nt = 0; nt < KT / 8; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const float p = exp2f(fmaf(s[nt][e], fl, mneg[e >> 1]));
            s[nt][e] = p;
            rsum[e >> 1] += p;
        }
#pragma unroll
    for (int r = 0; r < 2; ++r) lrow[r] = lrow[r] * corr[r] + rsum[r];
#pragma unroll
    for (int i = 0; i < NO; ++i) {
        o[i][0] *= corr[0]; o[i][1] *= corr[0];
        o[i][2] *= corr[1]; o[i][3] *= corr[1];
    }
}

constexpr float VD_LOG2E = 1.4426950408889634f;
__device__ __forceinline__ float vd_ex2(float x) {
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
    return r;
}
__device__ __forceinline__ float vd_rcp(float x) {
    float r;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
    return r;
}
// The score x (unscaled product) with soft cap c (0: none): c tanh(f x / c) = c - 2 c / (1 + e^(2 f x / c)), to an absolute error of a
// few 1e-7 c.  `two`: 2 f log2(e) / c.
__device__ __forceinline__ float vd_cap(float x, float f, float c, float two) {
    return c > 0.f ? fmaf(-2.f * c, vd_rcp(1.f + vd_ex2(x * two)), c) : x * f;
}
__device__ __forceinline__ float vd_sigmoid(float x) { return vd_rcp(1.f + vd_ex2(-VD_LOG2E * x)); }

template <int KT, int DV>
__device__ __forceinline__ void vd_pv(const float (&s)[KT / 8][4], float (&o)[DV / 8][4], const bf16* tV, int ldv, int lane) {
#pragma unroll
    for (int kt = 0; kt < KT / 16; ++kt) {
        uint32_t pa[4];
        pa[0] = pack_bf16(s[2 * kt][0], s[2 * kt][1]);
        pa[1] = pack_bf16(s[2 * kt][2], s[2 * kt][3]);
        pa[2] = pack_bf16(s[2 * kt + 1][0], s[2 * kt + 1][1]);
        pa[3] = pack_bf16(s[2 * kt + 1][2], s[2 * kt + 1][3]);
        const bf16* row = tV + (kt * 16 + (((lane >> 3) & 1) << 3) + (lane & 7)) * ldv + ((lane >> 4) << 3);
#pragma unroll
        for (int dt = 0; dt < DV / 16; ++dt) {
            uint32_t vb[4];
            ldsm_x4_t(vb, row + dt * 16);
            mma_bf16(o[2 * dt], pa, vb[0], vb[1]);
            mma_bf16(o[2 * dt + 1], pa, vb[2], vb[3]);
        }
    }
}

template <int KT>
__device__ __forceinline__ void vd_qk(float (&s)[KT / 8][4], const bf16* q16, int ldq, const bf16* tK, int ldk, int dk, int lane) {
#pragma unroll
    for (int i = 0; i < KT / 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
    const bf16* qrow = q16 + (lane & 15) * ldq + ((lane >> 4) << 3);
    const bf16* krow = tK + (((lane >> 4) << 3) + (lane & 7)) * ldk + (((lane >> 3) & 1) << 3);
#pragma unroll 4
    for (int kk = 0; kk < dk; kk += 16) {
        uint32_t qa[4];
        ldsm_x4(qa, qrow + kk);
#pragma unroll
        for (int nt = 0; nt < KT / 16; ++nt) {
            uint32_t kb[4];
            ldsm_x4(kb, krow + nt * 16 * ldk + kk);
            mma_bf16(s[2 * nt], qa, kb[0], kb[1]);
            mma_bf16(s[2 * nt + 1], qa, kb[2], kb[3]);
        }
    }
}

// ------------------------------------------------------------------------------------------
// Prefill: grid (query tiles, Hq, B), 128 threads.
// ------------------------------------------------------------------------------------------
template <int DV, int FORM>
__global__ void __launch_bounds__(128) attn_prefill_vd_kernel(AttnArgs a) {
    constexpr int BM = 64, BN = 64;
    constexpr bool FORMS = FORM > 0, EXT = FORM == 2;
    __shared__ float s_dist[EXT ? 128 : 1];          // what is added to the score, per distance of a tile (query row - key column + 63)
    pdl_wait();
    pdl_trigger();
    extern __shared__ __align__(128) unsigned char smem_raw[];
    const int dk = a.Dh, ldk = dk + 8, ldv = DV + 8, ck = dk / 8;
    constexpr int cv = DV / 8;
    bf16* sQ = reinterpret_cast<bf16*>(smem_raw);
    bf16* sK = sQ + BM * ldk;            // 2 stages
    bf16* sV = sK + 2 * BN * ldk;        // 2 stages

    const int b = blockIdx.z, h = blockIdx.y, hk = h / (a.Hq / a.Hkv);
    const int q0 = a.cu_q[b], qlen = a.cu_q[b + 1] - q0;
    const int m0 = (int)(gridDim.x - 1 - blockIdx.x) * BM;
    if (m0 >= qlen) return;
    const int kvlen = a.kv_lens[b];
    const int pos0 = a.q_pos0 ? a.q_pos0[b] : kvlen - qlen;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int rows = min(BM, qlen - m0);
    const int j_lo = a.window > 0 ? max(0, pos0 + m0 - a.window + 1) : 0;
    const int j_hi = min(pos0 + m0 + rows, kvlen);
    const int t_lo = j_lo / BN, t_hi = (j_hi + BN - 1) / BN;
    // tiles in order: those of the kept first positions that lie ahead of the window, then the window's
    const int n_first = FORMS && a.keep_first > 0 ? min(t_lo, (a.keep_first + BN - 1) / BN) : 0;
    const bool one_row = FORMS && a.kv_scale != 0;
    float* sF = reinterpret_cast<float*>(sV);                          // 2 stages of key factors, in place of the value tiles
    const float slope = FORMS && a.slopes ? a.slopes[h] : 0.f;
    const bool sig = EXT && a.sig_bias != nullptr;
    const float pb = sig ? a.sig_bias[h] : 0.f, r1 = EXT && a.log_r1 ? a.log_r1[h] : 0.f, r2 = EXT && a.log_r1 ? a.log_r2[h] : 0.f;
    const float cap2 = EXT && a.softcap > 0.f ? 2.f * VD_LOG2E * a.scale / a.softcap : 0.f;

    for (int i = threadIdx.x; i < BM * ck; i += 128) {
        const int r = i / ck, c = i % ck;
        bf16* dst = sQ + r * ldk + c * 8;
        if (r < rows) cp_async16(dst, a.q + ((long)(q0 + m0 + r) * a.Hq + h) * dk + c * 8);
        else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
    }
    // two threads per key row: each resolves the row's slot once and copies half of its pieces
    auto load_kv = [&](int t, int stage) {
        const int r = threadIdx.x >> 1, half = threadIdx.x & 1, j = t * BN + r;
        bf16* pk = sK + stage * BN * ldk + r * ldk;
        bf16* pv = sV + stage * BN * ldv + r * ldv;
        if (j < kvlen) {
            const long slot = vd_slot(a, b, j);
            const bf16* gk = a.k_cache + slot * a.k_ld + hk * dk;
            const bf16* gv = a.v_cache + slot * a.v_ld + hk * DV;
            for (int c = half; c < ck; c += 2) cp_async16(pk + c * 8, gk + c * 8);
            if (one_row) {
                if (half == 0) cp_async4(sF + stage * BN + r, attn_key_factor(a, slot));
                return;
            }
#pragma unroll
            for (int c = 0; c < cv; c += 2) cp_async16(pv + (c + half) * 8, gv + (c + half) * 8);
        } else {
            for (int c = half; c < ck; c += 2) *reinterpret_cast<uint4*>(pk + c * 8) = make_uint4(0, 0, 0, 0);
            if (one_row) {
                if (half == 0) sF[stage * BN + r] = 0.f;
                return;
            }
#pragma unroll
            for (int c = 0; c < cv; c += 2) *reinterpret_cast<uint4*>(pv + (c + half) * 8) = make_uint4(0, 0, 0, 0);
        }
    };
    load_kv(n_first > 0 ? 0 : t_lo, 0);
    cp_async_commit();

    float o[DV / 8][4];
#pragma unroll
    for (int i = 0; i < DV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    float mrow[2] = {-INFINITY, -INFINITY}, lrow[2] = {0.f, 0.f};
    const int r_lo = warp * 16 + (lane >> 2);
    const int qpos_a = pos0 + m0 + r_lo, qpos_b = qpos_a + 8;
    const int q_first = pos0 + m0 + warp * 16;

    for (int t = n_first > 0 ? 0 : t_lo, flip = 0; t < t_hi; t = FORMS && t + 1 == n_first ? t_lo : t + 1, flip ^= 1) {
        const int stage = FORMS ? flip : (t - t_lo) & 1, next = FORMS && t + 1 == n_first ? t_lo : t + 1;
        if (next < t_hi) load_kv(next, stage ^ 1);
        cp_async_commit();
        if (EXT) s_dist[threadIdx.x] = pb - r1 * log1pf(r2 * (float)max(0, pos0 + m0 - t * BN + (int)threadIdx.x - 63));
        cp_async_wait<1>();
        __syncthreads();
        float s[BN / 8][4];
        vd_qk<BN>(s, sQ + warp * 16 * ldk, ldk, sK + stage * BN * ldk, ldk, dk, lane);
        if (one_row) {
#pragma unroll
            for (int nt = 0; nt < BN / 8; ++nt) {
                const float2 kf = *reinterpret_cast<const float2*>(sF + stage * BN + nt * 8 + (lane & 3) * 2);
                s[nt][0] *= kf.x; s[nt][1] *= kf.y; s[nt][2] *= kf.x; s[nt][3] *= kf.y;
            }
        }
        float f = a.scale;
        if (EXT) {
            const float* dist = s_dist + r_lo - (lane & 3) * 2 + 63;
#pragma unroll
            for (int nt = 0; nt < BN / 8; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) s[nt][e] = vd_cap(s[nt][e], a.scale, a.softcap, cap2) + dist[(e < 2 ? 0 : 8) - nt * 8 - (e & 1)];
            f = 1.f;
        } else if (a.softcap > 0.f) {
            const float inv_cap = a.scale / a.softcap;
#pragma unroll
            for (int nt = 0; nt < BN / 8; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) s[nt][e] = a.softcap * tanhf(s[nt][e] * inv_cap);
            f = 1.f;
        }
        if (FORMS && a.slopes != nullptr) {
            const int d0 = t * BN + (lane & 3) * 2 - qpos_a;                        // key minus query
#pragma unroll
            for (int nt = 0; nt < BN / 8; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) s[nt][e] = fmaf(slope, (float)(d0 + nt * 8 + (e & 1) - (e < 2 ? 0 : 8)), s[nt][e] * f);
            f = 1.f;
        }
        const bool need_mask = (t * BN + BN - 1 > q_first) || ((t + 1) * BN > kvlen) ||
                               (a.window > 0 && t * BN <= q_first + 15 - a.window);
        if (need_mask) {
#pragma unroll
            for (int nt = 0; nt < BN / 8; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int j = t * BN + nt * 8 + (lane & 3) * 2 + (e & 1);
                    const int qp = (e < 2) ? qpos_a : qpos_b;
                    const bool ok = j <= qp && j < kvlen && (a.window <= 0 || j > qp - a.window || (FORMS && j < a.keep_first));
                    s[nt][e] = ok ? s[nt][e] : -INFINITY;
                }
        }
        if (sig) {
#pragma unroll
            for (int nt = 0; nt < BN / 8; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) s[nt][e] = vd_sigmoid(s[nt][e]);             // -inf: 0
        } else {
            vd_softmax<BN, DV / 8>(s, o, mrow, lrow, f);
        }
        vd_pv<BN, DV>(s, o, one_row ? sK + stage * BN * ldk : sV + stage * BN * ldv, ldv, lane);      // one row: ldk = ldv
        __syncthreads();
    }
    cp_async_wait<0>();
    float inv[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        lrow[r] += __shfl_xor_sync(0xffffffffu, lrow[r], 1);
        lrow[r] += __shfl_xor_sync(0xffffffffu, lrow[r], 2);
        float mm = mrow[r], ll = lrow[r], oc = 1.f;
        if (a.sinks) {
            const float sk = a.sinks[h], mn = fmaxf(mm, sk);
            oc = (mm == -INFINITY) ? 0.f : __expf(mm - mn);
            ll = ll * oc + __expf(sk - mn);
        }
        inv[r] = sig ? 1.f : ll > 0.f ? oc / ll : 0.f;
        const int row = r_lo + 8 * r;
        if (row < rows) {
            if (!FORMS || !a.gate_cols) inv[r] *= attn_gate(a, q0 + m0 + row, h);
            if (a.lse_out != nullptr && (lane & 3) == 0)
                a.lse_out[(long)(q0 + m0 + row) * a.Hq + h] = lrow[r] > 0.f ? mrow[r] + __logf(lrow[r]) : -INFINITY;
        }
    }
#pragma unroll
    for (int i = 0; i < DV / 8; ++i) {
        const int d = i * 8 + (lane & 3) * 2;
        if (FORMS && a.gate_cols) {
            const long t = q0 + m0 + r_lo;
            if (r_lo < rows) { o[i][0] *= attn_gate(a, t, h, d); o[i][1] *= attn_gate(a, t, h, d + 1); }
            if (r_lo + 8 < rows) { o[i][2] *= attn_gate(a, t + 8, h, d); o[i][3] *= attn_gate(a, t + 8, h, d + 1); }
        }
        if (r_lo < rows)
            *reinterpret_cast<uint32_t*>(a.out + ((long)(q0 + m0 + r_lo) * a.Hq + h) * DV + d) = pack_bf16(o[i][0] * inv[0], o[i][1] * inv[0]);
        if (r_lo + 8 < rows)
            *reinterpret_cast<uint32_t*>(a.out + ((long)(q0 + m0 + r_lo + 8) * a.Hq + h) * DV + d) = pack_bf16(o[i][2] * inv[1], o[i][3] * inv[1]);
    }
}

// ------------------------------------------------------------------------------------------
// Decode: grid (splits, Hkv * chunks, B), 128 threads; a CTA serves up to 16 query heads of one KV head.  Each warp walks
// its own 32-key pieces of the split.
// ------------------------------------------------------------------------------------------
template <int DV, int FORM>
__global__ void __launch_bounds__(128) attn_decode_vd_kernel(AttnArgs a, int chunks) {
    constexpr int KT = 32, cv = DV / 8;
    constexpr bool FORMS = FORM > 0, EXT = FORM == 2;
    pdl_wait();
    pdl_trigger();
    extern __shared__ __align__(128) unsigned char smem_raw[];
    const int dk = a.Dh, ldk = dk + 8, ldv = DV + 8, ck = dk / 8;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    bf16* sQ = reinterpret_cast<bf16*>(smem_raw);                       // [16][ldk]
    bf16* sK = sQ + 16 * ldk + warp * KT * (FORMS && a.kv_scale ? ldk : ldk + ldv);                 // this warp's K tile
    bf16* sV = sK + KT * ldk;                                           // and V tile
    const int split = blockIdx.x, hk = blockIdx.y / chunks, b = blockIdx.z;
    const int group = a.Hq / a.Hkv, first = (blockIdx.y % chunks) * 16;
    const int G = min(16, group - first), h0 = hk * group + first;

    for (int i = threadIdx.x; i < 16 * ck; i += 128) {
        const int r = i / ck, c = i % ck;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (r < G) v = *reinterpret_cast<const uint4*>(a.q + ((long)b * a.Hq + h0 + r) * dk + c * 8);
        *reinterpret_cast<uint4*>(sQ + r * ldk + c * 8) = v;
    }
    // the visible positions, numbered without a gap: the kept first ones ahead of the window, then the window
    const int len = a.kv_lens[b];
    const int lo = (a.window > 0 && len > a.window) ? len - a.window : 0, nf = FORMS ? min(a.keep_first, lo) : 0, gap = lo - nf;
    const int span = len - gap;
    const int per = a.split_len > 0 ? a.split_len : ((((span + a.splits - 1) / a.splits) + 31) & ~31);
    const int s0 = split * per, s1 = min(span, s0 + per);
    const bool one_row = FORMS && a.kv_scale != 0;
    float slope[2] = {0.f, 0.f};
    if (FORMS && a.slopes != nullptr) {
#pragma unroll
        for (int r = 0; r < 2; ++r)
            if ((lane >> 2) + 8 * r < G) slope[r] = a.slopes[h0 + (lane >> 2) + 8 * r];
    }
    const bool sig = EXT && a.sig_bias != nullptr;
    const float cap2 = EXT && a.softcap > 0.f ? 2.f * VD_LOG2E * a.scale / a.softcap : 0.f;
    float pb[2] = {0.f, 0.f}, r1[2] = {0.f, 0.f}, r2[2] = {0.f, 0.f};
    if (EXT) {
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int row = (lane >> 2) + 8 * r;
            if (row < G) {
                if (sig) pb[r] = a.sig_bias[h0 + row];
                if (a.log_r1 != nullptr) { r1[r] = a.log_r1[h0 + row]; r2[r] = a.log_r2[h0 + row]; }
            }
        }
    }
    __syncthreads();

    float o[DV / 8][4];
#pragma unroll
    for (int i = 0; i < DV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    float mrow[2] = {-INFINITY, -INFINITY}, lrow[2] = {0.f, 0.f};

    for (int base = s0 + warp * KT; base < s1; base += 4 * KT) {
        const int j = base + lane;
        const long slot = j < s1 ? vd_slot(a, b, j < nf ? j : j + gap) : 0;
        const float kf = one_row && j < s1 ? *attn_key_factor(a, slot) : 0.f;
        // consecutive lanes copy consecutive pieces of a row; rows past the end are zero
        for (int i = lane; i < KT * ck; i += 32) {
            const int key = i / ck, c = i % ck;
            const long sl = __shfl_sync(0xffffffffu, slot, key);
            bf16* p = sK + key * ldk + c * 8;
            if (base + key < s1) cp_async16(p, a.k_cache + sl * a.k_ld + hk * dk + c * 8);
            else *reinterpret_cast<uint4*>(p) = make_uint4(0u, 0u, 0u, 0u);
        }
        if (!one_row)
#pragma unroll 4
        for (int i = lane; i < KT * cv; i += 32) {
            const int key = i / cv, c = i % cv;
            const long sl = __shfl_sync(0xffffffffu, slot, key);
            bf16* p = sV + key * ldv + c * 8;
            if (base + key < s1) cp_async16(p, a.v_cache + sl * a.v_ld + hk * DV + c * 8);
            else *reinterpret_cast<uint4*>(p) = make_uint4(0u, 0u, 0u, 0u);
        }
        cp_async_commit();
        cp_async_wait<0>();
        __syncwarp();
        float s[KT / 8][4];
        vd_qk<KT>(s, sQ, ldk, sK, ldk, dk, lane);
        if (one_row) {
#pragma unroll
            for (int nt = 0; nt < KT / 8; ++nt) {
                const float k0 = __shfl_sync(0xffffffffu, kf, nt * 8 + (lane & 3) * 2), k1 = __shfl_sync(0xffffffffu, kf, nt * 8 + (lane & 3) * 2 + 1);
                s[nt][0] *= k0; s[nt][1] *= k1; s[nt][2] *= k0; s[nt][3] *= k1;
            }
        }
        float f = a.scale;
        if (EXT) {
#pragma unroll
            for (int nt = 0; nt < KT / 8; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int i = base + nt * 8 + (lane & 3) * 2 + (e & 1), r = e >> 1;
                    const float d = (float)max(0, len - 1 - (i < nf ? i : i + gap));
                    s[nt][e] = vd_cap(s[nt][e], a.scale, a.softcap, cap2) + (pb[r] - r1[r] * __logf(fmaf(r2[r], d, 1.f)));
                }
            f = 1.f;
        } else if (a.softcap > 0.f) {
#pragma unroll
            for (int nt = 0; nt < KT / 8; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) s[nt][e] = a.softcap * tanhf(s[nt][e] * a.scale / a.softcap);
            f = 1.f;
        }
        if (FORMS && a.slopes != nullptr) {
#pragma unroll
            for (int nt = 0; nt < KT / 8; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int i = base + nt * 8 + (lane & 3) * 2 + (e & 1);
                    s[nt][e] = fmaf(slope[e >> 1], (float)((i < nf ? i : i + gap) - (len - 1)), s[nt][e] * f);
                }
            f = 1.f;
        }
#pragma unroll
        for (int nt = 0; nt < KT / 8; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (base + nt * 8 + (lane & 3) * 2 + (e & 1) >= s1) s[nt][e] = -INFINITY;
        if (sig) {
#pragma unroll
            for (int nt = 0; nt < KT / 8; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) s[nt][e] = vd_sigmoid(s[nt][e]);
        } else {
            vd_softmax<KT, DV / 8>(s, o, mrow, lrow, f);
        }
        vd_pv<KT, DV>(s, o, one_row ? sK : sV, ldv, lane);
        __syncwarp();
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        lrow[r] += __shfl_xor_sync(0xffffffffu, lrow[r], 1);
        lrow[r] += __shfl_xor_sync(0xffffffffu, lrow[r], 2);
        if (sig) mrow[r] = 0.f;                                         // partial sums are added as they are
    }
    __syncthreads();
    float* red_m = reinterpret_cast<float*>(smem_raw);                  // [4][16]
    float* red_l = red_m + 64;                                          // [4][16]
    float* red_o = red_l + 64;                                          // [4][G][DV]
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const int row = (lane >> 2) + 8 * r;
        if (row < G) {
            if ((lane & 3) == 0) { red_m[warp * 16 + row] = mrow[r]; red_l[warp * 16 + row] = lrow[r]; }
#pragma unroll
            for (int i = 0; i < DV / 8; ++i) {
                float* dst = red_o + (warp * G + row) * DV + i * 8 + (lane & 3) * 2;
                dst[0] = o[i][2 * r];
                dst[1] = o[i][2 * r + 1];
            }
        }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < G * DV; i += 128) {
        const int g = i / DV, d = i % DV;
        float mm = -INFINITY, ll = 0.f, ov = 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w) mm = fmaxf(mm, red_m[w * 16 + g]);
#pragma unroll
        for (int w = 0; w < 4; ++w) {
            const float c = (red_m[w * 16 + g] == -INFINITY) ? 0.f : __expf(red_m[w * 16 + g] - mm);
            ll += red_l[w * 16 + g] * c;
            ov += red_o[(w * G + g) * DV + d] * c;
        }
        const long pi = ((long)b * a.Hq + h0 + g) * a.splits + split;
        a.part_o[pi * DV + d] = ov;
        // sigmoid weights: maxima 0 and a sum of 1 over all splits, so that the merge adds the parts as they are
        if (d == 0) { a.part_ml[pi * 2] = mm; a.part_ml[pi * 2 + 1] = !sig ? ll : split == 0 ? 1.f : 0.f; }
    }
}

template <int DV, int FORMS>
static int launch_vd_form(const AttnArgs& a, int max_q, cudaStream_t s) {
    const int ldk = a.Dh + 8, ldv = DV + 8;
    static bool configured = false;
    if (!configured) {
        TSB_CHECK_CUDA(cudaFuncSetAttribute(attn_prefill_vd_kernel<DV, FORMS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        TSB_CHECK_CUDA(cudaFuncSetAttribute(attn_decode_vd_kernel<DV, FORMS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        configured = true;
    }
    if (max_q > 0) {
        const size_t smem = (size_t)(64 * ldk + 2 * 64 * (a.kv_scale ? ldk + 2 : ldk + ldv)) * sizeof(bf16);       // (a factor per row: two elements)
        TSB_CHECK_CUDA(tsb_launch(attn_prefill_vd_kernel<DV, FORMS>, dim3((max_q + 63) / 64, a.Hq, a.B), dim3(128), smem, s, a));
    } else {
        const int chunks = (a.Hq / a.Hkv + 15) / 16;
        const size_t stage = (size_t)(16 * ldk + 4 * 32 * (a.kv_scale ? ldk : ldk + ldv)) * sizeof(bf16), merge = (size_t)(128 + 4 * 16 * DV) * sizeof(float);
        TSB_CHECK_CUDA(tsb_launch(attn_decode_vd_kernel<DV, FORMS>, dim3(a.splits, a.Hkv * chunks, a.B), dim3(128), stage > merge ? stage : merge, s,
                                  a, chunks));
    }
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}

template <int DV>
static int launch_vd(const AttnArgs& a, int max_q, cudaStream_t s) {
    if (a.log_r1 != nullptr || a.sig_bias != nullptr) return launch_vd_form<DV, 2>(a, max_q, s);
    const bool forms = a.keep_first > 0 || a.slopes != nullptr || a.gate_cols || a.kv_scale;
    return forms ? launch_vd_form<DV, 1>(a, max_q, s) : launch_vd_form<DV, 0>(a, max_q, s);
}

static int dispatch_vd(const AttnArgs& in, int max_q, cudaStream_t s) {
    AttnArgs a = in;
    if (a.Dv == 0) a.Dv = a.Dh;
    if (a.k_ld == 0) a.k_ld = (long)a.Hkv * a.Dh;
    if (a.v_ld == 0) a.v_ld = (long)a.Hkv * a.Dv;
    TSB_CHECK_ARG(a.kv_scale == 0 || (a.Dv == a.Dh && a.kv_scale % 2 == 0), "attention: rows of %d / %d elements are not key and value at once", a.Dh, a.Dv);
    TSB_CHECK_ARG(a.keep_first >= 0 && (a.keep_first == 0 || a.window > 0), "attention: kept first positions without a window");
    TSB_CHECK_ARG(a.sig_bias == nullptr || (a.sinks == nullptr && a.lse_out == nullptr), "attention: sigmoid weights have no sink and no log-sum-exp");
    TSB_CHECK_ARG((a.log_r1 == nullptr) == (a.log_r2 == nullptr), "attention: a logarithmic distance bias has two numbers per head");
    TSB_CHECK_ARG(a.split_len == 0 || a.window <= 0, "attention: fixed splits with a window");
    TSB_CHECK_ARG(a.k_ld % 8 == 0 && a.v_ld % 8 == 0, "attention: cache rows of %ld / %ld elements are not 16-byte aligned", a.k_ld, a.v_ld);
    if (a.Dh <= 0 || a.Dh > 256 || a.Dh % 16 || a.Dv <= 0 || a.Dv > 256 || a.Dv % 16) {
        tsb_set_error("attention: unsupported head sizes %d / %d (multiples of 16 up to 256, or 512 with equal sizes)", a.Dh, a.Dv);
        return TSB_ERR_UNSUPPORTED;
    }
    switch (a.Dv) {
    case 16: return launch_vd<16>(a, max_q, s);
    case 32: return launch_vd<32>(a, max_q, s);
    case 48: return launch_vd<48>(a, max_q, s);
    case 64: return launch_vd<64>(a, max_q, s);
    case 80: return launch_vd<80>(a, max_q, s);
    case 96: return launch_vd<96>(a, max_q, s);
    case 112: return launch_vd<112>(a, max_q, s);
    case 128: return launch_vd<128>(a, max_q, s);
    case 144: return launch_vd<144>(a, max_q, s);
    case 160: return launch_vd<160>(a, max_q, s);
    case 176: return launch_vd<176>(a, max_q, s);
    case 192: return launch_vd<192>(a, max_q, s);
    case 208: return launch_vd<208>(a, max_q, s);
    case 224: return launch_vd<224>(a, max_q, s);
    case 240: return launch_vd<240>(a, max_q, s);
    default: return launch_vd<256>(a, max_q, s);
    }
}

int tsb_attn_prefill_vd_launch(const AttnArgs& a, int max_q, cudaStream_t s) { return max_q > 0 ? dispatch_vd(a, max_q, s) : TSB_OK; }
int tsb_attn_decode_vd_launch(const AttnArgs& a, cudaStream_t s) { return dispatch_vd(a, 0, s); }
