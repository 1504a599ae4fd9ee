// Retention: a linear recurrence whose heads fade at constant rates g_h,
//
//   S_t = g_h S_(t-1) + k_t v_t^T       (S: [dk, dv] per head),       o_t = S_t^T q_t
//
// q and k are columns of a 32-bit projection, the first 2 * half dims of each head turned by the token's position (dim i
// with dim i + half), k then times a constant; v other columns of it.  Everything here is 32-bit.  The state lives per
// sequence as [H][dk][dv] and is carried from step to step.
//
// Steps of a few tokens per sequence walk them one by one (retention_walk_kernel).  Longer portions are cut into chunks
// of RT_C tokens that run side by side.  Over a chunk that starts from S_in, with n tokens counted from 0,
//
//   o_t   = g^(t+1) S_in^T q_t + sum_(s<=t) g^(t-s) (k_s . q_t) v_s
//   S_out = g^n S_in + sum_s g^(n-1-s) k_s v_s^T
//
// so the work is products of tiles: what a chunk adds to the state (retention_chunk_state_kernel), the chunks' states one
// after another (retention_carry_kernel: S_in of every chunk, from and to the sequence's state), and the read-outs
// (retention_chunk_out_kernel).  The sums are those of the walk in another order.  In front of them
// retention_turn_kernel turns q and k in place, once.
#include "common.cuh"

#define RT_C 64                 // tokens of a chunk
#define RT_LD 68                // row stride of a tile of 64 columns in shared memory (16-byte rows, banks spread)

struct RetentionArgs {
    float* proj; int stride, col_q, col_k, col_v;
    const float2* cs; int half;                     // [N, half] (cos, sin)
    float k_scale;
    const float* decay;                             // [H]
    float* state; long long state_stride;           // state + slot * stride : [H][dk][dv]
    float* o; int o_stride;                         // o[t, h * dv + j]
    const int* cu_q; const int* slots;
    const int* chunk_t0; const int* seq_chunk0;     // the chunks' first packed tokens [n_chunks + 1], each sequence's first chunk
    float* chunk_state;                             // [n_chunks][H][dk][dv]
    int H, dk, dv, n_tokens;
    int vec;                                        // tiles may be read in 16-byte pieces
};

// element d of a head's row x, turned by the token's row of the table
__device__ __forceinline__ float retention_turned(const float* __restrict__ x, int d, int half, const float2* __restrict__ cs) {
    if (d >= 2 * half) return x[d];
    const bool first = d < half;
    const float2 a = cs[first ? d : d - half];
    return first ? x[d] * a.x - x[d + half] * a.y : x[d] * a.x + x[d - half] * a.y;
}

// ------------------------------------------------------------------ few tokens per sequence: one after another
// A block has (sequence, head, 32 columns of S): warp w holds rows w, w + 8, .. of them in registers, a lane a column.
template <int RP>
__global__ void __launch_bounds__(256) retention_walk_kernel(RetentionArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float qk[2][8 * RP];
    __shared__ float part[8][32];
    const int s = blockIdx.z, h = blockIdx.y, w = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int j = blockIdx.x * 32 + lane;
    const bool col = j < a.dv;
    const int t0 = a.cu_q[s], t1 = a.cu_q[s + 1];
    float* sp = a.state + (size_t)a.slots[s] * a.state_stride + (size_t)h * a.dk * a.dv + (col ? j : 0);
    const float g = a.decay[h];
    float S[RP];
#pragma unroll
    for (int i = 0; i < RP; ++i) S[i] = (col && w + 8 * i < a.dk) ? sp[(size_t)(w + 8 * i) * a.dv] : 0.f;
    for (int t = t0; t < t1; ++t) {
        const float* row = a.proj + (size_t)t * a.stride;
        const float2* cs = a.cs + (size_t)t * a.half;
        const float v = col ? row[a.col_v + h * a.dv + j] : 0.f;
        for (int e = threadIdx.x; e < 2 * 8 * RP; e += 256) {
            const int which = e / (8 * RP), d = e % (8 * RP);
            float x = 0.f;
            if (d < a.dk) {
                x = retention_turned(row + (which ? a.col_k : a.col_q) + h * a.dk, d, a.half, cs);
                if (which) x *= a.k_scale;
            }
            qk[which][d] = x;
        }
        __syncthreads();
        float acc = 0.f;
#pragma unroll
        for (int i = 0; i < RP; ++i) {
            S[i] = fmaf(qk[1][w + 8 * i], v, g * S[i]);
            acc = fmaf(S[i], qk[0][w + 8 * i], acc);
        }
        part[w][lane] = acc;
        __syncthreads();
        if (w == 0 && col) {
            float y = 0.f;
#pragma unroll
            for (int p = 0; p < 8; ++p) y += part[p][lane];
            a.o[(size_t)t * a.o_stride + h * a.dv + j] = y;
        }
    }
#pragma unroll
    for (int i = 0; i < RP; ++i)
        if (col && w + 8 * i < a.dk) sp[(size_t)(w + 8 * i) * a.dv] = S[i];
}

// ------------------------------------------------------------------ long portions
// q and k turned in place, k times its constant: a thread per pair (or untouched dim) of a head
__global__ void __launch_bounds__(256) retention_turn_kernel(RetentionArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, per = a.dk - a.half;
    float* row = a.proj + (size_t)t * a.stride;
    for (int e = blockIdx.y * blockDim.x + threadIdx.x; e < 2 * a.H * per; e += gridDim.y * blockDim.x) {
        const int which = e / (a.H * per), h = e % (a.H * per) / per, i = e % per;
        float* x = row + (which ? a.col_k : a.col_q) + h * a.dk;
        const float f = which ? a.k_scale : 1.f;
        if (i < a.half) {
            const float2 cs = a.cs[(size_t)t * a.half + i];
            const float u = x[i], v = x[i + a.half];
            x[i] = (u * cs.x - v * cs.y) * f;
            x[i + a.half] = (v * cs.x + u * cs.y) * f;
        } else if (which) {
            x[i + a.half] *= f;
        }
    }
}

__device__ __forceinline__ void rt_copy16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
// a tile of 64 x 64 floats into shared memory (row stride RT_LD): rows r < n_rows at src + r * ld, columns c < n_cols;
// zeros elsewhere.  16-byte copies are asynchronous: rt_wait() before the barrier that hands the tile over.
__device__ __forceinline__ void rt_tile(float* dst, const float* __restrict__ src, size_t ld, int n_rows, int n_cols, int vec) {
    if (vec) {
        for (int e = threadIdx.x; e < 64 * 16; e += 256) {
            const int r = e >> 4, c = (e & 15) * 4;
            float* to = dst + r * RT_LD + c;
            if (r < n_rows && c < n_cols) rt_copy16(to, src + (size_t)r * ld + c);
            else *reinterpret_cast<float4*>(to) = make_float4(0.f, 0.f, 0.f, 0.f);
        }
    } else {
        for (int e = threadIdx.x; e < 64 * 64; e += 256) {
            const int r = e >> 6, c = e & 63;
            dst[r * RT_LD + c] = (r < n_rows && c < n_cols) ? src[(size_t)r * ld + c] : 0.f;
        }
    }
}
__device__ __forceinline__ void rt_wait() { asm volatile("cp.async.wait_all;\n" ::: "memory"); }

// chunk_state[c, h, d, j] = sum_s g^(n-1-s) k_s[d] v_s[j]: a block per (chunk, head, 64 DT x 64 of the state), 4 DT x 4 of
// them a thread (two tiles of dims share the values' reads)
#define RT_STATE_SMEM(DT) (((DT) + 1) * RT_C * RT_LD * (int)sizeof(float))
template <int DT>
__global__ void __launch_bounds__(256) retention_chunk_state_kernel(RetentionArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) float sm[];
    float* sv = sm;
    float* sk = sv + RT_C * RT_LD;                   // [DT] tiles
    __shared__ float pw[RT_C];
    const int c = blockIdx.x, h = blockIdx.y, tiles_j = (a.dv + 63) / 64;
    const int d0 = blockIdx.z / tiles_j * (64 * DT), j0 = blockIdx.z % tiles_j * 64;
    const int t0 = a.chunk_t0[c], n = a.chunk_t0[c + 1] - t0;
    const float* base = a.proj + (size_t)t0 * a.stride;
#pragma unroll
    for (int m = 0; m < DT; ++m)
        rt_tile(sk + m * RT_C * RT_LD, base + a.col_k + h * a.dk + d0 + 64 * m, a.stride, n, min(64, a.dk - d0 - 64 * m), a.vec);
    rt_tile(sv, base + a.col_v + h * a.dv + j0, a.stride, n, min(64, a.dv - j0), a.vec);
    if (threadIdx.x < n) pw[threadIdx.x] = powf(a.decay[h], (float)(n - 1 - threadIdx.x));
    rt_wait();
    __syncthreads();
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
    float acc[DT][4][4];
#pragma unroll
    for (int m = 0; m < DT; ++m)
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int k = 0; k < 4; ++k) acc[m][i][k] = 0.f;
#pragma unroll 4
    for (int t = 0; t < n; ++t) {
        float4 v4 = *reinterpret_cast<const float4*>(sv + t * RT_LD + tx * 4);
        const float f = pw[t];
        const float vx[4] = {v4.x * f, v4.y * f, v4.z * f, v4.w * f};
#pragma unroll
        for (int m = 0; m < DT; ++m) {
            const float4 k4 = *reinterpret_cast<const float4*>(sk + (m * RT_C + t) * RT_LD + ty * 4);
            const float kx[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int k = 0; k < 4; ++k) acc[m][i][k] = fmaf(kx[i], vx[k], acc[m][i][k]);
        }
    }
    float* dst = a.chunk_state + ((size_t)c * a.H + h) * a.dk * a.dv;
#pragma unroll
    for (int m = 0; m < DT; ++m)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int d = d0 + 64 * m + ty * 4 + i, j = j0 + tx * 4;
            if (d >= a.dk) break;
            float* p = dst + (size_t)d * a.dv + j;
            if (a.vec && j + 4 <= a.dv) {
                *reinterpret_cast<float4*>(p) = make_float4(acc[m][i][0], acc[m][i][1], acc[m][i][2], acc[m][i][3]);
            } else {
#pragma unroll
                for (int k = 0; k < 4; ++k)
                    if (j + k < a.dv) p[k] = acc[m][i][k];
            }
        }
}

// chunk after chunk: what a chunk starts from takes the place of what it adds, and the state moves on.  A thread has V
// elements side by side; the chunks of a batch are on their way together, only the sums are a chain.
#define RT_BATCH 8
template <int V>
__global__ void __launch_bounds__(128) retention_carry_kernel(RetentionArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const int s = blockIdx.z, h = blockIdx.y;
    const size_t per = (size_t)a.dk * a.dv, e = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * V;
    if (e >= per) return;                                       // (V == 4: dv is a multiple of 4)
    const int c0 = a.seq_chunk0[s], c1 = a.seq_chunk0[s + 1];
    float* st = a.state + (size_t)a.slots[s] * a.state_stride + (size_t)h * per + e;
    float* cs = a.chunk_state + ((size_t)c0 * a.H + h) * per + e;
    const size_t step = (size_t)a.H * per;
    const float g = a.decay[h], whole = powf(g, (float)RT_C);
    // every chunk of a portion but its last is whole
    const float last = c1 > c0 ? powf(g, (float)(a.chunk_t0[c1] - a.chunk_t0[c1 - 1])) : 1.f;
    float S[V];
#pragma unroll
    for (int i = 0; i < V; ++i) S[i] = st[i];
    for (int b = c0; b < c1; b += RT_BATCH, cs += RT_BATCH * step) {
        float add[RT_BATCH][V];
#pragma unroll
        for (int u = 0; u < RT_BATCH; ++u)
            if (b + u < c1) {
                if constexpr (V == 4) {
                    const float4 x = *reinterpret_cast<const float4*>(cs + u * step);
                    add[u][0] = x.x; add[u][1] = x.y; add[u][2] = x.z; add[u][3] = x.w;
                } else add[u][0] = cs[u * step];
            }
#pragma unroll
        for (int u = 0; u < RT_BATCH; ++u)
            if (b + u < c1) {
                if constexpr (V == 4) *reinterpret_cast<float4*>(cs + u * step) = make_float4(S[0], S[1], S[2], S[3]);
                else cs[u * step] = S[0];
                const float f = b + u + 1 < c1 ? whole : last;
#pragma unroll
                for (int i = 0; i < V; ++i) S[i] = fmaf(f, S[i], add[u][i]);
            }
    }
#pragma unroll
    for (int i = 0; i < V; ++i) st[i] = S[i];
}

// read-outs: a block per (chunk, head, 64 columns); per 64 dims of the keys it adds q k^T to the chunk's pair scores and
// q S_in to its outputs (thread: 4 tokens x 4), then the masked and decayed scores times v
#define RT_OUT_SMEM (4 * RT_C * RT_LD * (int)sizeof(float))
__global__ void __launch_bounds__(256) retention_chunk_out_kernel(RetentionArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) float sm[];
    float* sq = sm;                                  // [tokens][dims]; the pair scores [t][s] once the dims are through
    float* sk = sq + RT_C * RT_LD;                   // [tokens][dims]
    float* ss = sk + RT_C * RT_LD;                   // [dims][columns]
    float* sv = ss + RT_C * RT_LD;                   // [tokens][columns]
    __shared__ float pw[RT_C + 1];
    const int c = blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * 64;
    const int t0 = a.chunk_t0[c], n = a.chunk_t0[c + 1] - t0, nj = min(64, a.dv - j0);
    const float* base = a.proj + (size_t)t0 * a.stride;
    const float* S = a.chunk_state + ((size_t)c * a.H + h) * a.dk * a.dv + j0;
    if (threadIdx.x <= RT_C) pw[threadIdx.x] = powf(a.decay[h], (float)threadIdx.x);
    rt_tile(sv, base + a.col_v + h * a.dv + j0, a.stride, n, nj, a.vec);
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
    const int nk = (4 * (ty | 1) + 3) / 16 + 1;      // groups of 16 tokens that a warp's rows (two ty) may see
    float pair[4][4], out[4][4];                     // pair[i][k]: tokens t = 4 ty + i, s = tx + 16 k;  out[i][k]: column 4 tx + k
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int k = 0; k < 4; ++k) pair[i][k] = out[i][k] = 0.f;
    for (int d0 = 0; d0 < a.dk; d0 += 64) {
        const int nd = min(64, a.dk - d0);
        if (d0) __syncthreads();
        rt_tile(sq, base + a.col_q + h * a.dk + d0, a.stride, n, nd, a.vec);
        rt_tile(sk, base + a.col_k + h * a.dk + d0, a.stride, n, nd, a.vec);
        rt_tile(ss, S + (size_t)d0 * a.dv, a.dv, nd, nj, a.vec);
        rt_wait();
        __syncthreads();
#pragma unroll 2
        for (int d = 0; d < 64; d += 4) {
            float4 q4[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) q4[i] = *reinterpret_cast<const float4*>(sq + (4 * ty + i) * RT_LD + d);
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                if (k >= nk) break;                  // (a warp's rows all lie before these tokens)
                const float4 k4 = *reinterpret_cast<const float4*>(sk + (tx + 16 * k) * RT_LD + d);
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    pair[i][k] = fmaf(q4[i].x, k4.x, pair[i][k]); pair[i][k] = fmaf(q4[i].y, k4.y, pair[i][k]);
                    pair[i][k] = fmaf(q4[i].z, k4.z, pair[i][k]); pair[i][k] = fmaf(q4[i].w, k4.w, pair[i][k]);
                }
            }
#pragma unroll
            for (int dd = 0; dd < 4; ++dd) {
                const float4 s4 = *reinterpret_cast<const float4*>(ss + (d + dd) * RT_LD + 4 * tx);
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const float q = dd == 0 ? q4[i].x : dd == 1 ? q4[i].y : dd == 2 ? q4[i].z : q4[i].w;
                    out[i][0] = fmaf(q, s4.x, out[i][0]); out[i][1] = fmaf(q, s4.y, out[i][1]);
                    out[i][2] = fmaf(q, s4.z, out[i][2]); out[i][3] = fmaf(q, s4.w, out[i][3]);
                }
            }
        }
    }
    __syncthreads();                                 // everyone is through with q: the scores take its place
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = 4 * ty + i;
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const int s = tx + 16 * k;
            sq[t * RT_LD + s] = s <= t ? pair[i][k] * pw[t - s] : 0.f;
            out[i][k] *= pw[t + 1];
        }
    }
    __syncthreads();
#pragma unroll 2
    for (int s = 0; s < 4 * ty + 4; s += 4) {        // (tokens behind a row's own have weight 0)
        float4 p4[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) p4[i] = *reinterpret_cast<const float4*>(sq + (4 * ty + i) * RT_LD + s);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const float4 v4 = *reinterpret_cast<const float4*>(sv + (s + e) * RT_LD + 4 * tx);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float p = e == 0 ? p4[i].x : e == 1 ? p4[i].y : e == 2 ? p4[i].z : p4[i].w;
                out[i][0] = fmaf(p, v4.x, out[i][0]); out[i][1] = fmaf(p, v4.y, out[i][1]);
                out[i][2] = fmaf(p, v4.z, out[i][2]); out[i][3] = fmaf(p, v4.w, out[i][3]);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = 4 * ty + i;
        if (t >= n) break;
        float* p = a.o + (size_t)(t0 + t) * a.o_stride + h * a.dv + j0 + 4 * tx;
        if (a.vec && 4 * tx + 4 <= nj) {
            *reinterpret_cast<float4*>(p) = make_float4(out[i][0], out[i][1], out[i][2], out[i][3]);
        } else {
#pragma unroll
            for (int k = 0; k < 4; ++k)
                if (4 * tx + k < nj) p[k] = out[i][k];
        }
    }
}

extern "C" int idm_retention_chunk_tokens() { return RT_C; }
// floats of scratch for a step of so many chunks
extern "C" long long idm_retention_scratch_floats(int n_chunks, int H, int dk, int dv) { return (long long)n_chunks * H * dk * dv; }

// chunk_t0 [n_chunks + 1], seq_chunk0 [n_seqs + 1] as for the other chunked recurrence (a chunk ends where the next
// begins, chunks hold RT_C tokens, a sequence's last one up to so many, and never cross a sequence's border); n_chunks == 0: every sequence token by
// token.  In chunks, the step's q and k columns of `proj` are turned in place.
extern "C" int idm_retention(float* proj, int stride, int col_q, int col_k, int col_v, const float* cs, int half, float k_scale,
                             const float* decay, float* state, long long state_stride, float* o, int o_stride, const int* cu_q,
                             const int* slots, int n_seqs, int H, int dk, int dv, const int* chunk_t0, const int* seq_chunk0,
                             int n_chunks, float* scratch, int n_tokens, cudaStream_t stream) {
    if (n_seqs == 0 || n_tokens == 0) return 0;
    IDM_REQUIRE(H > 0 && dk > 0 && dk <= 256 && dv > 0, "retention: %d heads, keys of %d (at most 256), values of %d", H, dk, dv);
    IDM_REQUIRE(half >= 0 && 2 * half <= dk && (half == 0 || cs != nullptr), "retention: %d turning pairs in heads of %d", half, dk);
    IDM_REQUIRE(col_q >= 0 && col_k >= 0 && col_v >= 0 && col_q + H * dk <= stride && col_k + H * dk <= stride && col_v + H * dv <= stride,
                "retention: columns beyond rows of %d", stride);
    IDM_REQUIRE(state != nullptr && state_stride >= (long long)H * dk * dv, "retention: a slot's state must hold %d x %d x %d floats", H, dk, dv);
    IDM_REQUIRE(n_seqs <= 65535 && H <= 65535, "retention: %d sequences, %d heads in one launch", n_seqs, H);
    IDM_REQUIRE(n_chunks == 0 || (chunk_t0 && seq_chunk0 && scratch), "retention: chunks need their lists and scratch");
    RetentionArgs a;
    a.proj = proj; a.stride = stride; a.col_q = col_q; a.col_k = col_k; a.col_v = col_v; a.cs = (const float2*)cs; a.half = half;
    a.k_scale = k_scale; a.decay = decay; a.state = state; a.state_stride = state_stride; a.o = o; a.o_stride = o_stride;
    a.cu_q = cu_q; a.slots = slots; a.chunk_t0 = chunk_t0; a.seq_chunk0 = seq_chunk0; a.chunk_state = scratch;
    a.H = H; a.dk = dk; a.dv = dv; a.n_tokens = n_tokens;
    a.vec = dk % 4 == 0 && dv % 4 == 0 && stride % 4 == 0 && col_q % 4 == 0 && col_k % 4 == 0 && col_v % 4 == 0 && o_stride % 4 == 0 &&
            (((uintptr_t)proj | (uintptr_t)scratch | (uintptr_t)o) & 15) == 0;
    if (n_chunks == 0) {
        const dim3 grid((dv + 31) / 32, H, n_seqs);
        if (dk <= 32) idm_launch(retention_walk_kernel<4>, grid, dim3(256), 0, stream, a);
        else if (dk <= 64) idm_launch(retention_walk_kernel<8>, grid, dim3(256), 0, stream, a);
        else if (dk <= 128) idm_launch(retention_walk_kernel<16>, grid, dim3(256), 0, stream, a);
        else idm_launch(retention_walk_kernel<32>, grid, dim3(256), 0, stream, a);
        IDM_LAUNCH_CHECK("retention_walk");
        return 0;
    }
    const int items = 2 * H * (dk - half), tiles_d = (dk + 63) / 64, tiles_j = (dv + 63) / 64;
    idm_launch(retention_turn_kernel, dim3(n_tokens, min(8, (items + 255) / 256)), dim3(256), 0, stream, a);
    IDM_LAUNCH_CHECK("retention_turn");
    static bool set = false;
    if (!set) {
        cudaError_t e = cudaFuncSetAttribute(retention_chunk_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, RT_OUT_SMEM);
        if (e == cudaSuccess)
            e = cudaFuncSetAttribute(retention_chunk_state_kernel<2>, cudaFuncAttributeMaxDynamicSharedMemorySize, RT_STATE_SMEM(2));
        IDM_REQUIRE(e == cudaSuccess, "retention: %d bytes of shared memory were refused (%s)", RT_OUT_SMEM, cudaGetErrorString(e));
        set = true;
    }
    if (tiles_d > 1)
        idm_launch(retention_chunk_state_kernel<2>, dim3(n_chunks, H, (tiles_d + 1) / 2 * tiles_j), dim3(256), RT_STATE_SMEM(2), stream, a);
    else
        idm_launch(retention_chunk_state_kernel<1>, dim3(n_chunks, H, tiles_j), dim3(256), RT_STATE_SMEM(1), stream, a);
    IDM_LAUNCH_CHECK("retention_chunk_state");
    const size_t per = (size_t)dk * dv;
    if (a.vec)
        idm_launch(retention_carry_kernel<4>, dim3((unsigned)((per / 4 + 127) / 128), H, n_seqs), dim3(128), 0, stream, a);
    else
        idm_launch(retention_carry_kernel<1>, dim3((unsigned)((per + 127) / 128), H, n_seqs), dim3(128), 0, stream, a);
    IDM_LAUNCH_CHECK("retention_carry");
    idm_launch(retention_chunk_out_kernel, dim3(n_chunks, H, tiles_j), dim3(256), RT_OUT_SMEM, stream, a);
    IDM_LAUNCH_CHECK("retention_chunk_out");
    return 0;
}
