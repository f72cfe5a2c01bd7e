// Residual streams side by side (hyper-connections), and the norm that needs no statistics.
//
// A model may carry S copies of its residual stream, x_1 .. x_S, instead of one.  A sublayer reads a weighted sum of
// them, u = sum_s in[s] x_s, and afterwards every stream is made anew from all the old ones and the sublayer's output:
// x_t <- sum_s mix[s, t] x_s + out[t] y.  Both are the same work for every coordinate, and so is the norm
// tanh(alpha u) * w + b, so ONE pass over the streams applies the update that the sublayer before left pending, writes
// the streams, and hands the next sublayer its normed input.  With S = 1 and coefficients of one it is "add, then norm"
// of an ordinary residual stream.
//
//   source   x [T, S, d], or - before anything was written - ONE row per token that all streams equal (base [T, d])
//   update   none; y FP32 [T, d]; or the rows that routed experts left, y[t] = sum_j weights[t, j] z[row of pair (t, j)]
//   read     in [S] (null: all ones, the plain sum of the streams)
//   norm     alpha, w, b -> the activations' type; null: u itself, FP32
//   rows     null: every row, streams written back; else the output rows are the given ones and nothing is written back
//
// Streams, sums, coefficients and the norm are FP32.
#include "common.cuh"

#define HY_THREADS 128
#define HY_MAX_STREAMS 32

struct HyArgs {
    float* x;                    // [T, S, d]
    const float* base;           // [T, d] or null
    int S, d, n_rows, write_back;
    int update;                  // 0 none, 1 y, 2 routed rows
    const float* y;
    const void* z;
    const int* ids;
    const float* weights;
    const int* row_of_pair;      // null: pair p's row is p
    int top, all_experts;
    const float* mix;            // [S, S], from x to
    const float* out;            // [S]
    const float* in;             // [S] or null
    const float* alpha;          // [1], w [d], b [d]: or null
    const float* w;
    const float* b;
    void* h;                     // the output rows: T with a norm, FP32 without
    const int* rows;
};

template <int V> __device__ __forceinline__ void hy_load(const float* p, float* v) {
    if (V == 4) NiVec16<float>::load(p, v);
    else
#pragma unroll
        for (int k = 0; k < V; ++k) v[k] = p[k];
}
template <int V> __device__ __forceinline__ void hy_store(float* p, const float* v) {
    if (V == 4) NiVec16<float>::store(p, v);
    else
#pragma unroll
        for (int k = 0; k < V; ++k) p[k] = v[k];
}
template <typename T, int V> __device__ __forceinline__ void hy_load_act(const T* p, float* v) {
#pragma unroll
    for (int k = 0; k < V; ++k) v[k] = ni_to_float(p[k]);
}
template <> __device__ __forceinline__ void hy_load_act<float, 4>(const float* p, float* v) { NiVec16<float>::load(p, v); }
template <> __device__ __forceinline__ void hy_load_act<__nv_bfloat16, 4>(const __nv_bfloat16* p, float* v) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}
template <typename T, int V> __device__ __forceinline__ void hy_store_act(T* p, const float* v) {
#pragma unroll
    for (int k = 0; k < V; ++k) p[k] = ni_from_float<T>(v[k]);
}
template <> __device__ __forceinline__ void hy_store_act<float, 4>(float* p, const float* v) { NiVec16<float>::store(p, v); }
template <> __device__ __forceinline__ void hy_store_act<__nv_bfloat16, 4>(__nv_bfloat16* p, const float* v) {
    uint2 raw;
    *reinterpret_cast<__nv_bfloat162*>(&raw.x) = __floats2bfloat162_rn(v[0], v[1]);
    *reinterpret_cast<__nv_bfloat162*>(&raw.y) = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = raw;
}

// grid (column pieces of HY_THREADS * V, row lanes): a block walks rows of one column piece, coefficients in shared
// memory, the norm's weight and bias in registers.  MS: the most streams this instance takes (S <= MS).
template <typename T, int MS, int V>
__global__ void __launch_bounds__(HY_THREADS) hyper_step_kernel(const HyArgs a) {
    __shared__ float s_mix[MS * MS], s_out[MS], s_in[MS];
    const int S = a.S;
    for (int i = threadIdx.x; i < MS * MS; i += HY_THREADS) {
        const int from = i / MS, to = i - from * MS;
        s_mix[i] = (a.update && from < S && to < S) ? a.mix[from * S + to] : 0.f;
    }
    for (int i = threadIdx.x; i < MS; i += HY_THREADS) {
        s_out[i] = (a.update && i < S) ? a.out[i] : 0.f;
        s_in[i] = i < S ? (a.in ? a.in[i] : 1.0f) : 0.f;
    }
    __syncthreads();
    const int c = (blockIdx.x * HY_THREADS + threadIdx.x) * V;
    if (c >= a.d) return;
    const size_t d = a.d;
    float w[V], b[V];
    const float alpha = a.alpha ? a.alpha[0] : 0.f;
    if (a.alpha) {
        hy_load<V>(a.w + c, w);
        hy_load<V>(a.b + c, b);
    }
    for (int i = blockIdx.y; i < a.n_rows; i += gridDim.y) {
        const size_t t = a.rows ? a.rows[i] : i;
        float x[MS][V];
        if (a.base) {
            float one[V];
            hy_load<V>(a.base + t * d + c, one);
#pragma unroll
            for (int s = 0; s < MS; ++s)
#pragma unroll
                for (int k = 0; k < V; ++k) x[s][k] = one[k];
        } else {
#pragma unroll
            for (int s = 0; s < MS; ++s)
                if (s < S) hy_load<V>(a.x + (t * S + s) * d + c, x[s]);
                else
#pragma unroll
                    for (int k = 0; k < V; ++k) x[s][k] = 0.f;
        }
        float u[V];
#pragma unroll
        for (int k = 0; k < V; ++k) u[k] = 0.f;
        if (a.update) {
            float y[V];
            if (a.update == 1) {
                hy_load<V>(a.y + t * d + c, y);
            } else {
#pragma unroll
                for (int k = 0; k < V; ++k) y[k] = 0.f;
                // four rows at a time: their numbers, then the rows, are on their way together
                for (int j0 = 0; j0 < a.top; j0 += 4) {
                    size_t row[4];
                    float wgt[4], zv[4][V];
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        const size_t p = t * a.top + min(j0 + j, a.top - 1);
                        row[j] = a.all_experts > 0 ? t * a.all_experts + a.ids[p] : (a.row_of_pair ? (size_t)a.row_of_pair[p] : p);
                        wgt[j] = a.weights[p];
                    }
#pragma unroll
                    for (int j = 0; j < 4; ++j) hy_load_act<T, V>(reinterpret_cast<const T*>(a.z) + row[j] * d + c, zv[j]);
#pragma unroll
                    for (int j = 0; j < 4; ++j)
                        if (j0 + j < a.top)
#pragma unroll
                            for (int k = 0; k < V; ++k) y[k] = fmaf(wgt[j], zv[j][k], y[k]);
                }
            }
#pragma unroll
            for (int to = 0; to < MS; ++to) {
                if (to >= S) break;
                float v[V];
#pragma unroll
                for (int k = 0; k < V; ++k) v[k] = s_out[to] * y[k];
#pragma unroll
                for (int s = 0; s < MS; ++s) {
                    if (MS > 8 && s >= S) break;
                    const float m = s_mix[s * MS + to];
#pragma unroll
                    for (int k = 0; k < V; ++k) v[k] = fmaf(m, x[s][k], v[k]);
                }
                if (a.write_back) hy_store<V>(a.x + (t * S + to) * d + c, v);
                const float in = s_in[to];
#pragma unroll
                for (int k = 0; k < V; ++k) u[k] = fmaf(in, v[k], u[k]);
            }
        } else {
#pragma unroll
            for (int s = 0; s < MS; ++s)
#pragma unroll
                for (int k = 0; k < V; ++k) u[k] = fmaf(s_in[s], x[s][k], u[k]);
        }
        if (a.alpha) {
#pragma unroll
            for (int k = 0; k < V; ++k) u[k] = fmaf(tanhf(alpha * u[k]), w[k], b[k]);
            hy_store_act<T, V>(reinterpret_cast<T*>(a.h) + (size_t)i * d + c, u);
        } else if (a.h) {
            hy_store<V>(reinterpret_cast<float*>(a.h) + (size_t)i * d + c, u);
        }
    }
}

template <typename T, int MS, int V>
static int launch_hyper(const HyArgs& a, cudaStream_t stream) {
    const int pieces = (a.d + HY_THREADS * V - 1) / (HY_THREADS * V);
    const int most = (16 * ni_sm_count() + pieces - 1) / pieces;           // blocks that are resident at once, about
    dim3 grid(pieces, a.n_rows < most ? a.n_rows : most);
    if (grid.y > 65535) grid.y = 65535;
    hyper_step_kernel<T, MS, V><<<grid, HY_THREADS, 0, stream>>>(a);
    NI_RETURN_LAUNCH_STATUS();
}

template <typename T>
static int dispatch_hyper(const HyArgs& a, bool vec, cudaStream_t stream) {
    if (a.S > 8) return launch_hyper<T, HY_MAX_STREAMS, 1>(a, stream);
    if (vec) {
        if (a.S == 1) return launch_hyper<T, 1, 4>(a, stream);
        if (a.S == 2) return launch_hyper<T, 2, 4>(a, stream);
        if (a.S == 3) return launch_hyper<T, 3, 4>(a, stream);
        if (a.S == 4) return launch_hyper<T, 4, 4>(a, stream);
        return launch_hyper<T, 8, 4>(a, stream);
    }
    if (a.S <= 2) return launch_hyper<T, 2, 1>(a, stream);
    if (a.S <= 4) return launch_hyper<T, 4, 1>(a, stream);
    return launch_hyper<T, 8, 1>(a, stream);
}

NI_EXPORT int ni_hyper_max_streams() { return HY_MAX_STREAMS; }

// See the head of this file; act_dtype: the type of z and of the normed output.
NI_EXPORT int ni_hyper_step(float* x, const float* base, int S, int d, int n_rows, int write_back, int update, const float* y,
                            const void* z, int act_dtype, const int* ids, const float* weights, const int* row_of_pair, int top,
                            int all_experts, const float* mix, const float* out, const float* in, const float* alpha,
                            const float* w, const float* b, void* h, const int* rows, cudaStream_t stream) {
    if (n_rows <= 0) return NI_OK;
    if (S <= 0 || d <= 0 || (!x && !base) || update < 0 || update > 2) return NI_ERR_BAD_ARGUMENT;
    if (S > HY_MAX_STREAMS) return NI_ERR_UNSUPPORTED_SIZE;
    if (update && (!mix || !out)) return NI_ERR_BAD_ARGUMENT;
    if (update == 1 && !y) return NI_ERR_BAD_ARGUMENT;
    if (update == 2 && (!z || !ids || !weights || top <= 0)) return NI_ERR_BAD_ARGUMENT;
    if (write_back && (!x || rows || !update)) return NI_ERR_BAD_ARGUMENT;
    if (alpha && (!w || !b || !h)) return NI_ERR_BAD_ARGUMENT;
    const HyArgs a = {x, base, S, d, n_rows, write_back, update, y, z, ids, weights, row_of_pair, top, all_experts,
                      mix, out, in, alpha, w, b, h, rows};
    const size_t bits = (size_t)x | (size_t)base | (size_t)y | (size_t)z | (size_t)w | (size_t)b | (size_t)h;
    const bool vec = d % 4 == 0 && (bits & 15) == 0;
    if (act_dtype == NI_DTYPE_F32) return dispatch_hyper<float>(a, vec, stream);
    if (act_dtype == NI_DTYPE_BF16) return dispatch_hyper<__nv_bfloat16>(a, vec, stream);
    return NI_ERR_BAD_ARGUMENT;
}
