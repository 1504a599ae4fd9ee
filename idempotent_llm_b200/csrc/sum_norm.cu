// RMS norm in groups, and the pass of a layer whose norm takes the stream and a sublayer's output together.
//
//   N(v): the row in `groups` equal parts of neighbours, each part over sqrt(mean(part^2) + eps), times w     (32-bit)
//   sum_norm:      h[r] <- N(alpha * h[r] + sum_p y[p][r])  stored, and x[r] = the same row in the storage type
//   grouped norm:  x[i] = N(h[rows[i]] + sum_p y[p][rows[i]])  for picked rows, the stream left alone
//
// A part of a row is worked on by a warp (up to 1024 elements) or by a block (more), whatever the number of rows: a
// row's bits depend on the row alone.
#include "common.cuh"

struct SumNormArgs {
    float* h; const float* y; int n_partials; size_t partial_stride;
    float alpha; const float* w; float eps;
    T* x;                        // or null
    const int* rows;             // or null
    int store;                   // the normed row replaces the stream's (never with `rows`)
    int n_parts;                 // rows * groups
    int hidden, groups, part;    // part = hidden / groups
};

__device__ __forceinline__ float4 sn_load4(const SumNormArgs& a, size_t at) {
    float4 v = *reinterpret_cast<const float4*>(a.h + at);
    v.x *= a.alpha; v.y *= a.alpha; v.z *= a.alpha; v.w *= a.alpha;
    for (int p = 0; p < a.n_partials; ++p) {
        const float4 u = __ldg(reinterpret_cast<const float4*>(a.y + (size_t)p * a.partial_stride + at));
        v.x += u.x; v.y += u.y; v.z += u.z; v.w += u.w;
    }
    return v;
}
__device__ __forceinline__ float sn_sumsq(const float4& v) { return fmaf(v.x, v.x, v.y * v.y) + fmaf(v.z, v.z, v.w * v.w); }

// NV groups of four neighbours per thread; THREADS of them share a part (a warp, or a block of 256)
template <int NV, bool WARP>
__global__ void __launch_bounds__(256) sum_norm_kernel(SumNormArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float scratch[32];
    const int lanes = WARP ? 32 : 256, lane = WARP ? threadIdx.x & 31 : threadIdx.x;
    const int seg = WARP ? blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5) : blockIdx.x;
    if (seg >= a.n_parts) return;                       // (whole warps; a block-wide launch has exactly n_parts blocks)
    const int i = seg / a.groups, col0 = (seg % a.groups) * a.part;
    const size_t from = (size_t)(a.rows ? a.rows[i] : i) * a.hidden + col0, to = (size_t)i * a.hidden + col0;
    float4 v[NV];
    float s = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int c = (lanes * k + lane) * 4;
        v[k] = c < a.part ? sn_load4(a, from + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int k = 0; k < NV; ++k) s += sn_sumsq(v[k]);
    s = WARP ? warp_sum(s) : block_sum(s, scratch);
    const float inv = 1.0f / sqrtf(s / (float)a.part + a.eps);
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int c = (lanes * k + lane) * 4;
        if (c < a.part) {
            const float4 wv = __ldg(reinterpret_cast<const float4*>(a.w + col0 + c));
            const float4 o = make_float4(v[k].x * inv * wv.x, v[k].y * inv * wv.y, v[k].z * inv * wv.z, v[k].w * inv * wv.w);
            if (a.store) *reinterpret_cast<float4*>(a.h + from + c) = o;
            if (a.x) store4(a.x + to + c, o.x, o.y, o.z, o.w);
        }
    }
}

// parts of any length (element by element, the part waiting in shared memory between the passes)
__global__ void __launch_bounds__(256) sum_norm_any_kernel(SumNormArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float scratch[32];
    extern __shared__ float vals[];
    const int seg = blockIdx.x, i = seg / a.groups, col0 = (seg % a.groups) * a.part;
    const size_t from = (size_t)(a.rows ? a.rows[i] : i) * a.hidden + col0, to = (size_t)i * a.hidden + col0;
    float s = 0.f;
    for (int c = threadIdx.x; c < a.part; c += blockDim.x) {
        const float v = add_partials(a.h[from + c] * a.alpha, a.y, a.n_partials, a.partial_stride, from + c);
        vals[c] = v;
        s = fmaf(v, v, s);
    }
    const float inv = 1.0f / sqrtf(block_sum(s, scratch) / (float)a.part + a.eps);
    for (int c = threadIdx.x; c < a.part; c += blockDim.x) {
        const float o = vals[c] * inv * a.w[col0 + c];
        if (a.store) a.h[from + c] = o;
        if (a.x) from_f32(a.x[to + c], o);
    }
}

// rows == null: n_rows rows of the stream; store: they are replaced.  rows != null: x[i] of row rows[i], nothing stored.
extern "C" int idm_sum_norm(float* h, const float* y, int n_partials, long long partial_stride, float alpha, const float* w,
                            float eps, int groups, void* x, const int* rows, int store, int n_rows, int hidden,
                            cudaStream_t stream) {
    if (n_rows == 0) return 0;
    IDM_REQUIRE(hidden > 0 && n_rows > 0 && groups >= 1 && hidden % groups == 0, "sum_norm: rows=%d hidden=%d groups=%d", n_rows, hidden, groups);
    IDM_REQUIRE(!(store && rows) && (store || x != nullptr), "sum_norm: picked rows leave the stream alone, and something is written");
    SumNormArgs a;
    a.h = h; a.y = y; a.n_partials = y ? n_partials : 0; a.partial_stride = (size_t)partial_stride; a.alpha = alpha; a.w = w; a.eps = eps;
    a.x = (T*)x; a.rows = rows; a.store = store; a.hidden = hidden; a.groups = groups; a.part = hidden / groups;
    IDM_REQUIRE((long long)n_rows * groups < (1ll << 30), "sum_norm: %d rows of %d parts in one step", n_rows, groups);
    a.n_parts = n_rows * groups;
    if (a.part % 4 == 0 && a.part <= 1024) {
        const int per = a.n_parts >= 64 ? 8 : 1;        // warps (parts) a block: the arithmetic of a part is the same
        const dim3 grid((unsigned)((a.n_parts + per - 1) / per)), block(32 * per);
        if (a.part <= 256) idm_launch(sum_norm_kernel<2, true>, grid, block, 0, stream, a);
        else if (a.part <= 512) idm_launch(sum_norm_kernel<4, true>, grid, block, 0, stream, a);
        else idm_launch(sum_norm_kernel<8, true>, grid, block, 0, stream, a);
    } else if (a.part % 4 == 0 && a.part <= 4096) {
        if (a.part <= 2048) idm_launch(sum_norm_kernel<2, false>, dim3((unsigned)a.n_parts), dim3(256), 0, stream, a);
        else idm_launch(sum_norm_kernel<4, false>, dim3((unsigned)a.n_parts), dim3(256), 0, stream, a);
    } else {
        const size_t smem = (size_t)a.part * sizeof(float);
        IDM_REQUIRE(smem <= 160 * 1024, "sum_norm: parts of %d do not fit shared memory", a.part);
        if (smem > 48 * 1024) cudaFuncSetAttribute(sum_norm_any_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        idm_launch(sum_norm_any_kernel, dim3((unsigned)a.n_parts), dim3(256), smem, stream, a);
    }
    IDM_LAUNCH_CHECK("sum_norm");
    return 0;
}
