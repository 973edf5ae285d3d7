// The 32-bit forms of the matrix products and of attention, for models that run in float32 (compute_dtype float32): plain
// FMA arithmetic, no tensor-core mode.  Weights stay in their stored type (bf16 or f32) and are widened as they are read.
#include "attn_args.cuh"
#include "common.cuh"

// ------------------------------------------------------------------------------------------
// out[t, n] = sum_k X[x(t), k] W[n, k] (+ bias[n]).  64 x 64 tiles, 256 threads, 4 x 4 outputs per thread, K slabs of 16.
// Grouped (tiles != null): W is a stack of matrices of N rows, tile y of the grid is {matrix or -1, first row, end row}.
// Row t reads X row rows[t] / row_div when `rows` is given (the sorted (token, slot) pairs of a mixture of experts).
// ------------------------------------------------------------------------------------------
struct GemmF32Args {
    const void* W; const float* X; float* out; const float* bias;
    const int* tiles; const int* rows;
    long ldx, ldo;
    int T, N, K, row_div;
};

template <typename TW>
__global__ void __launch_bounds__(256) gemm_f32_kernel(GemmF32Args a) {
    __shared__ float sx[16][68], sw[16][68];
    pdl_wait();
    pdl_trigger();
    int t0 = blockIdx.y * 64, t_end = a.T;
    long w0 = 0;
    if (a.tiles != nullptr) {
        const int* g = a.tiles + 3 * blockIdx.y;
        if (g[0] < 0) return;
        w0 = (long)g[0] * a.N;
        t0 = g[1];
        t_end = g[2];
    }
    const int n0 = blockIdx.x * 64;
    const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;            // row and first k this thread stages
    const bool x_ok = t0 + lr < t_end, w_ok = n0 + lr < a.N;
    long xrow = x_ok ? t0 + lr : 0;
    if (x_ok && a.rows != nullptr) xrow = a.rows[xrow] / a.row_div;
    const float* xp = a.X + xrow * a.ldx;
    const TW* wp = reinterpret_cast<const TW*>(a.W) + (w0 + (w_ok ? n0 + lr : 0)) * a.K;
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    for (int k0 = 0; k0 < a.K; k0 += 16) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int k = k0 + lk + i;
            sx[lk + i][lr] = (x_ok && k < a.K) ? xp[k] : 0.f;
            sw[lk + i][lr] = (w_ok && k < a.K) ? (float)wp[k] : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < 16; ++k) {
            float xv[4], wv[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) { xv[i] = sx[k][ty * 4 + i]; wv[i] = sw[k][tx * 4 + i]; }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xv[i], wv[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = t0 + ty * 4 + i;
        if (t >= t_end) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int n = n0 + tx * 4 + j;
            if (n < a.N) a.out[(long)t * a.ldo + n] = acc[i][j] + (a.bias ? a.bias[n] : 0.f);
        }
    }
}

extern "C" int tsb_gemm_f32(const GemmF32Args* args, int w_bf16, int n_tiles, void* stream) {
    const GemmF32Args& a = *args;
    TSB_CHECK_ARG(a.T >= 0 && a.N > 0 && a.K > 0 && a.row_div > 0, "gemm_f32: bad shape T=%d N=%d K=%d", a.T, a.N, a.K);
    const int ty = a.tiles != nullptr ? n_tiles : (a.T + 63) / 64;
    TSB_CHECK_ARG(ty <= 65535, "gemm_f32: %d row tiles exceed the grid limit", ty);
    if (a.T == 0 || ty == 0) return TSB_OK;
    const dim3 grid((a.N + 63) / 64, ty);
    cudaStream_t s = (cudaStream_t)stream;
    if (w_bf16) TSB_CHECK_CUDA(tsb_launch(gemm_f32_kernel<bf16>, grid, dim3(256), 0, s, a));
    else TSB_CHECK_CUDA(tsb_launch(gemm_f32_kernel<float>, grid, dim3(256), 0, s, a));
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}

// ------------------------------------------------------------------------------------------
// Attention over a paged f32 cache, prompts and decode alike: grid (T, Hq), one CTA of four warps per (query row, head),
// each warp takes every fourth group of 32 keys (lane = key for the scores, lane = columns lane, lane + 32, .. for P V).
// q [T, Hq, Dh], k_cache [slots, Hkv, Dh], v_cache [slots, Hkv, Dv], out [T, Hq, Dv]; the pointers of AttnArgs hold floats.
// ------------------------------------------------------------------------------------------
#define ATTN_F32_MAX_DV 512

__global__ void __launch_bounds__(128) attn_f32_kernel(AttnArgs a) {
    constexpr int NJ = ATTN_F32_MAX_DV / 32;
    extern __shared__ float sm[];
    float* sq = sm;                              // [Dh]
    float* so = sm + a.Dh;                       // [4][Dv]
    __shared__ float sml[4][2];
    pdl_wait();
    pdl_trigger();
    const int t = blockIdx.x, h = blockIdx.y, hk = h / (a.Hq / a.Hkv);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    int b = 0;
    while (b + 1 < a.B && t >= a.cu_q[b + 1]) ++b;
    const float* kc = reinterpret_cast<const float*>(a.k_cache);
    const float* vc = reinterpret_cast<const float*>(a.v_cache);
    const float* q = reinterpret_cast<const float*>(a.q) + ((long)t * a.Hq + h) * a.Dh;
    for (int d = threadIdx.x; d < a.Dh; d += 128) sq[d] = q[d];
    __syncthreads();
    const int pos = a.kv_lens[b] - (a.cu_q[b + 1] - t);                   // this row's position
    // the visible positions, numbered without a gap: the kept first ones ahead of the window, then the window
    const int lo = a.window > 0 ? max(0, pos - a.window + 1) : 0, nf = min(a.keep_first, lo), gap = lo - nf, last = pos - gap;
    const float slope = a.slopes ? a.slopes[h] : 0.f;
    const bool one_row = a.kv_scale != 0, sig = a.sig_bias != nullptr;
    const float pb = sig ? a.sig_bias[h] : 0.f, r1 = a.log_r1 ? a.log_r1[h] : 0.f, r2 = a.log_r1 ? a.log_r2[h] : 0.f;
    float m = sig ? 0.f : -INFINITY, l = 0.f, acc[NJ];
#pragma unroll
    for (int j = 0; j < NJ; ++j) acc[j] = 0.f;
    for (int base = warp * 32; base <= last; base += 128) {
        const int i = base + lane, j = i < nf ? i : i + gap;
        const bool ok = i <= last;
        const long slot = ok ? (long)a.block_table[(long)b * a.max_pages + j / a.page_size] * a.page_size + j % a.page_size : 0;
        float s = -INFINITY;
        if (ok) {
            s = 0.f;
            const float* kp = kc + slot * a.k_ld + hk * a.Dh;
            for (int d = 0; d < a.Dh; ++d) s = fmaf(sq[d], kp[d], s);
            if (one_row) s *= kc[slot * a.k_ld + a.kv_scale];
            s *= a.scale;
            if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
            s = fmaf(slope, (float)(j - pos), s);
            if (a.log_r1 != nullptr) s -= r1 * log1pf(r2 * (float)(pos - j));
        }
        const float mx = sig ? 0.f : fmaxf(m, warp_max(s));
        const float corr = m == -INFINITY ? 0.f : sig ? 1.f : expf(m - mx);
        const float p = !ok ? 0.f : sig ? 1.f / (1.f + expf(-(s + pb))) : expf(s - mx);
        l = l * corr + warp_sum(p);
        m = mx;
#pragma unroll
        for (int i = 0; i < NJ; ++i) acc[i] *= corr;
        const int cnt = min(32, last - base + 1);
        for (int u = 0; u < cnt; ++u) {
            const float pu = __shfl_sync(0xffffffffu, p, u);
            const long su = __shfl_sync(0xffffffffu, slot, u);
            const float* vp = one_row ? kc + su * a.k_ld + hk * a.Dh : vc + su * a.v_ld + hk * a.Dv;
#pragma unroll
            for (int i = 0; i < NJ; ++i) {
                const int d = lane + 32 * i;
                if (d < a.Dv) acc[i] = fmaf(pu, vp[d], acc[i]);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < NJ; ++i) {
        const int d = lane + 32 * i;
        if (d < a.Dv) so[warp * a.Dv + d] = acc[i];
    }
    if (lane == 0) { sml[warp][0] = m; sml[warp][1] = l; }
    __syncthreads();
    float mm = a.sinks ? a.sinks[h] : -INFINITY;
    for (int w = 0; w < 4; ++w) mm = fmaxf(mm, sml[w][0]);
    float ll = a.sinks ? expf(a.sinks[h] - mm) : 0.f, c[4];
    for (int w = 0; w < 4; ++w) {
        c[w] = sml[w][0] == -INFINITY ? 0.f : expf(sml[w][0] - mm);
        ll += sml[w][1] * c[w];
    }
    if (sig) ll = 1.f;                           // weights that are not normalised
    float g = 1.f;
    const float* gate = reinterpret_cast<const float*>(a.gate);
    if (gate != nullptr && !a.gate_cols) g = 1.f / (1.f + expf(-gate[(long)t * a.gate_tok + h]));
    float* out = reinterpret_cast<float*>(a.out) + ((long)t * a.Hq + h) * a.Dv;
    for (int d = threadIdx.x; d < a.Dv; d += 128) {
        const float o = so[d] * c[0] + so[a.Dv + d] * c[1] + so[2 * a.Dv + d] * c[2] + so[3 * a.Dv + d] * c[3];
        if (a.gate_cols) g = 1.f / (1.f + expf(-gate[(long)t * a.gate_tok + h * a.Dv + d]));
        out[d] = o / ll * g;
    }
}

extern "C" int tsb_attn_f32(const AttnArgs* args, int T, void* stream) {
    AttnArgs a = *args;
    if (a.Dv == 0) a.Dv = a.Dh;
    if (a.k_ld == 0) a.k_ld = (long)a.Hkv * a.Dh;
    if (a.v_ld == 0) a.v_ld = (long)a.Hkv * a.Dv;
    TSB_CHECK_ARG(a.Hkv > 0 && a.Hq % a.Hkv == 0 && a.cu_q != nullptr, "attn_f32: Hq=%d Hkv=%d", a.Hq, a.Hkv);
    TSB_CHECK_ARG(a.Dh > 0 && a.Dh <= 1024 && a.Dv > 0 && a.Dv <= ATTN_F32_MAX_DV, "attn_f32: head sizes %d / %d", a.Dh, a.Dv);
    TSB_CHECK_ARG(a.kv_scale == 0 || a.Dv == a.Dh, "attn_f32: rows of %d / %d elements are not key and value at once", a.Dh, a.Dv);
    TSB_CHECK_ARG(a.sig_bias == nullptr || a.sinks == nullptr, "attn_f32: sigmoid weights have no sink");
    TSB_CHECK_ARG((a.log_r1 == nullptr) == (a.log_r2 == nullptr), "attn_f32: a logarithmic distance bias has two numbers per head");
    TSB_CHECK_ARG(a.gate != nullptr || !a.gate_cols, "attn_f32: no gate given");
    TSB_CHECK_ARG(a.gate == nullptr || a.gate_f32, "attn_f32: the gate must be float32");
    if (T == 0) return TSB_OK;
    cudaStream_t s = (cudaStream_t)stream;
    TSB_CHECK_CUDA(tsb_launch(attn_f32_kernel, dim3(T, a.Hq), dim3(128), (size_t)(a.Dh + 4 * a.Dv) * sizeof(float), s, a));
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}
