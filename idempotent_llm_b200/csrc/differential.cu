// The combination of a differential attention's two maps, behind the attention itself: a head has two contexts over the
// same values, a1 and a2 (rows 2 h and 2 h + 1 of o), and goes on as
//
//   o = a1 - lambda a2;   o / sqrt(mean(o^2) + eps) * post * sigmoid(gate[t, h])        (gate null: no gate)
//
// lambda and post are constants of the layer.  All of it in 32-bit, one warp per (token, head); nothing depends on the
// step's other tokens.
#include "common.cuh"

#define DF_WARPS 4
#define DF_MAX (IDM_MAX_HEAD_DIM / 32)

template <bool PAIRS>
__global__ void __launch_bounds__(DF_WARPS * 32) diff_combine_kernel(const T* __restrict__ o, float lambda, float eps, float post,
                                                                     const float* __restrict__ gate, int gate_stride,
                                                                     T* __restrict__ out, int out_stride, int out_col,
                                                                     int n_tokens, int H, int dv) {
    pdl_launch_dependents();
    pdl_wait();
    const long long i = (long long)blockIdx.x * DF_WARPS + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    if (i >= (long long)n_tokens * H) return;                   // whole warps leave; no block barrier below
    const int t = (int)(i / H), h = (int)(i % H);
    const T* a1 = o + (size_t)i * 2 * dv;
    const T* a2 = a1 + dv;
    T* dst = out + (size_t)t * out_stride + out_col + (size_t)h * dv;
    float x[DF_MAX], ss = 0.f;
    // PAIRS: a lane has neighbours 2 lane, 2 lane + 1 of every 64 elements, else element lane of every 32
#pragma unroll
    for (int e = 0; e < DF_MAX; ++e) {
        const int d = PAIRS ? (e >> 1) * 64 + 2 * lane + (e & 1) : e * 32 + lane;
        x[e] = d < dv ? fmaf(-lambda, to_f32(a2[d]), to_f32(a1[d])) : 0.f;
        ss = fmaf(x[e], x[e], ss);
    }
    float f = post / sqrtf(warp_sum(ss) / (float)dv + eps);
    if (gate) f = f / (1.0f + expf(-gate[(size_t)t * gate_stride + h]));
#pragma unroll
    for (int e = 0; e < DF_MAX; ++e) {
        const int d = PAIRS ? (e >> 1) * 64 + 2 * lane + (e & 1) : e * 32 + lane;
        if (d < dv) from_f32(dst[d], x[e] * f);
    }
}

extern "C" int idm_diff_combine(const void* o, float lambda, float eps, float post, const float* gate, int gate_stride, void* out,
                                int out_stride, int out_col, int n_tokens, int n_heads, int dv, cudaStream_t stream) {
    if (n_tokens == 0) return 0;
    IDM_REQUIRE(n_heads > 0 && dv > 0 && dv <= IDM_MAX_HEAD_DIM, "diff_combine: %d heads of %d (at most %d)", n_heads, dv, IDM_MAX_HEAD_DIM);
    IDM_REQUIRE(out_col >= 0 && out_col + n_heads * dv <= out_stride, "diff_combine: columns %d..%d of rows of %d", out_col,
                out_col + n_heads * dv, out_stride);
    IDM_REQUIRE(gate == nullptr || gate_stride >= n_heads, "diff_combine: %d gates in rows of %d", n_heads, gate_stride);
    const long long warps = (long long)n_tokens * n_heads;
    const dim3 grid((unsigned)((warps + DF_WARPS - 1) / DF_WARPS)), block(DF_WARPS * 32);
    if (dv % 2 == 0)
        idm_launch(diff_combine_kernel<true>, grid, block, 0, stream, (const T*)o, lambda, eps, post, gate, gate_stride, (T*)out,
                   out_stride, out_col, n_tokens, n_heads, dv);
    else
        idm_launch(diff_combine_kernel<false>, grid, block, 0, stream, (const T*)o, lambda, eps, post, gate, gate_stride, (T*)out,
                   out_stride, out_col, n_tokens, n_heads, dv);
    IDM_LAUNCH_CHECK("diff_combine");
    return 0;
}
