// Small-batch matrix-vector product over bf16 weights: the contract of gemv_kernel (gemv.cu) without the tensor-parallel
// push, in a kernel of its own.  gemv_kernel carries the decoders of every block format and their registers (over 100 per
// thread, four CTAs per SM); with bf16 rows alone a thread needs half of them, so twice as many warps stream weights.
// One warp per output row (with a gated activation: per gate / up row pair), four 16-byte loads per row and lane in flight
// (dot_bf16 in gemv_core.cuh).  Sums run in the same order for every M, so a row's result does not depend on the batch.
#include "gemv_core.cuh"

template <int M, bool GLU>
__global__ void __launch_bounds__(128) gemv_bf16_kernel(GemvArgs a) {
    const int lane = threadIdx.x & 31, r = blockIdx.x * 4 + (threadIdx.x >> 5), p = blockIdx.y;
    if (r >= a.n_out) return;
    int expert = 0, xrow = p * M, orow = p * M;
    if (a.ids) {
        pdl_wait();                                 // expert ids come from the router kernel
        pdl_trigger();
        expert = a.ids[p];
        if (expert < 0) return;
        xrow = p / a.x_div;
        orow = p;
    }
    const int mv = a.ids ? 1 : min(M, a.M - orow);
    const bf16* xb = a.xb + (long)xrow * a.w.K;
    const long wrow = (long)expert * a.w.N + r;
    float acc[M], acc2[M];
#pragma unroll
    for (int m = 0; m < M; ++m) { acc[m] = 0.f; acc2[m] = 0.f; }
    if (GLU) {
        const long rows[2] = {wrow, wrow + a.n_out};
        float* const out[2] = {acc, acc2};
        dot_bf16<M, 2>(a.w, rows, lane, xb, out, mv, PdlWait{a.ids == nullptr});
    } else {
        const long rows[1] = {wrow};
        float* const out[1] = {acc};
        dot_bf16<M, 1>(a.w, rows, lane, xb, out, mv, PdlWait{a.ids == nullptr});
    }
#pragma unroll
    for (int m = 0; m < M; ++m) {
        acc[m] = warp_sum(acc[m]);
        if (GLU) acc2[m] = warp_sum(acc2[m]);
    }
    if (lane != 0) return;
#pragma unroll
    for (int m = 0; m < M; ++m) {
        if (m >= mv) break;
        float v = acc[m];
        if (a.bias) v += a.bias[wrow];
        if (GLU) {
            v = act_glu(a.act, v, acc2[m] + (a.bias ? a.bias[wrow + a.n_out] : 0.f), expert < a.n_first ? a.lim_first : a.lim);
        } else if (a.act == ACT_RELU2) {
            v = fmaxf(v, 0.f);
            v = v * v;
        }
        if (a.row_scale) v *= a.row_scale[orow + m];
        const long o = (long)(orow + m) * a.n_out + r;
        if (a.out_f32) {
            if (a.residual) v += reinterpret_cast<const float*>(a.residual)[o];
            reinterpret_cast<float*>(a.out)[o] = v;
        } else {
            if (a.residual) v += bf2f(reinterpret_cast<const bf16*>(a.residual)[o]);
            reinterpret_cast<bf16*>(a.out)[o] = f2bf(v);
        }
    }
}

bool tsb_gemv_bf16_eligible(const GemvArgs& a) { return a.w.type == TSB_BF16 && a.push == nullptr && a.xb != nullptr && a.act != ACT_SILU; }

int tsb_gemv_bf16_launch(const GemvArgs& a, bool glu, int problems, cudaStream_t s) {
    const int M = a.ids ? 1 : a.M, rows = (a.n_out + 3) / 4;
    const dim3 block(128), grid(rows, a.ids ? problems : (M + 7) / 8);
#define TSB_GEMV_BF16(MM)                                                                          \
    {                                                                                              \
        if (glu) TSB_CHECK_CUDA(tsb_launch(gemv_bf16_kernel<MM, true>, grid, block, 0, s, a));     \
        else TSB_CHECK_CUDA(tsb_launch(gemv_bf16_kernel<MM, false>, grid, block, 0, s, a));        \
    }
    if (M <= 1) TSB_GEMV_BF16(1)
    else if (M <= 2) TSB_GEMV_BF16(2)
    else if (M <= 4) TSB_GEMV_BF16(4)
    else TSB_GEMV_BF16(8)
#undef TSB_GEMV_BF16
    TSB_CHECK_LAUNCH();
    return TSB_OK;
}
