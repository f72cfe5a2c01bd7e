// What lies between the fused q | k | v projection and the attention of a mixer whose queries and keys are
// normed as a whole: per token, in FP32 whatever the tensors' type,
//
//   q, k, v  += bias                         (optional; one FP32 vector over the projection's columns)
//   q <- q / sqrt(mean(q^2) + eps) * gain    over ALL H * D query values at once, and likewise the G * D key
//                                            values (optional; gains FP32 [H D] and [G D])
//   rotation of the first `rotary_dim` dimensions of every head of q and k, dimension i paired with
//            i + rotary_dim / 2:  (u, v) -> (u c - v s, v c + u s),  c = m cos(a), s = m sin(a),
//            a = float(position) * inv_freq[i]  (m = `magnitude`: an encoding that also scales what it rotates)
//   (optional, `head_unit`) every head of q and of k divided by its own root mean square over D, eps inside the
//            root, no weight - after the rotation
//   (optional, temp_coef) q <- q * (1 + temp_coef * ln(1 + floor((position + 1) / temp_every))): a factor on the finished
//            query that grows with the position
//   (optional, first_v) v <- (1 - lambda) v + lambda (first + first_bias): another layer's values of the same token, as
//            that layer's projection holds them, mixed in
//   q -> q_out [T, H D];  k -> key pages [P, G, page, D];  v -> value pages [P, G, page, V]
//
// One block per token.  The row's queries and keys are widened once into shared memory, where the two sums of
// squares and the partner of every rotated dimension are found; the angles' cosines and sines are computed
// once per token and shared by all heads.  The projection may be FP32 where queries and pages are bfloat16.
#include "common.cuh"

// What the options need beyond sizes and tables.
template <typename TI> struct QkExtra {
    float temp_coef, temp_every;      // temp_coef 0: no factor
    const TI* first_v;                // the other layer's value columns [T, first_ld], or null
    int first_ld;
    const float* first_bias;          // [G V] or null
    float lambda;
};
__device__ __forceinline__ float qk_temperature(float coef, float every, int pos) {
    return coef == 0.f ? 1.f : 1.f + coef * logf(floorf((float)(pos + 1) / every) + 1.f);
}
// VEC neighbouring numbers of a row (16-byte aligned), widened.
template <typename T, int VEC> __device__ __forceinline__ void qk_load(const T* p, float* v) {
#pragma unroll
    for (int k = 0; k < VEC; k += NiVec16<T>::N) NiVec16<T>::load(p + k, v + k);
}

// The heads' own norms: vals [(H + G) D] in shared memory holds the token's finished queries and keys; a warp takes
// a head at a time, divides it by its root mean square and writes it out (a key only where there are pages).
template <typename T>
__device__ __forceinline__ void qk_head_unit_write(const float* __restrict__ vals, float eps, float temp, T* __restrict__ q_row,
                                                   T* __restrict__ kdst, int H, int G, int D, int page_size) {
    __syncthreads();
    const int lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    for (int head = threadIdx.x >> 5; head < H + G; head += warps) {
        const float* x = vals + (size_t)head * D;
        float ss = 0.f;
        for (int d = lane; d < D; d += 32) ss = fmaf(x[d], x[d], ss);
        ss = ni_warp_sum(ss);
        const float inv = (head < H ? temp : 1.0f) / sqrtf(ss / (float)D + eps);
        T* dst = head < H ? q_row + (size_t)head * D : (kdst ? kdst + (size_t)(head - H) * page_size * D : nullptr);
        if (dst)
            for (int d = lane; d < D; d += 32) dst[d] = ni_from_float<T>(x[d] * inv);
    }
}

template <typename TI, typename T>
__global__ void __launch_bounds__(256)
qk_norm_rope_kernel(const TI* __restrict__ qkv, int ld, const float* __restrict__ bias,
                    const float* __restrict__ q_gain, const float* __restrict__ k_gain, float eps,
                    const int* __restrict__ positions, const int* __restrict__ seq_of_token,
                    const int* __restrict__ block_table, int bt_stride, const float* __restrict__ inv_freq,
                    float magnitude, T* __restrict__ q_out, T* __restrict__ k_pages, T* __restrict__ v_pages,
                    int H, int G, int D, int V, int rotary_dim, int page_size, int head_unit, const QkExtra<TI> ex) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float scratch[32];
    const int nq = H * D, nk = G * D, nv = G * V, half = rotary_dim >> 1;
    float* row = sm;                 // [nq + nk]: queries, then keys, bias added
    float* cs = sm + nq + nk;        // [2 half]: m cos, then m sin
    const int t = blockIdx.x;
    const TI* x = qkv + (size_t)t * ld;
    const int pos = positions[t];
    const float temp = qk_temperature(ex.temp_coef, ex.temp_every, pos);
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x; i < nq + nk; i += blockDim.x) {
        const float v = ni_to_float(x[i]) + (bias ? bias[i] : 0.f);
        row[i] = v;
        if (i < nq) sq += v * v; else sk += v * v;
    }
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        float s, c;
        sincosf((float)pos * inv_freq[i], &s, &c);
        cs[i] = c * magnitude;
        cs[half + i] = s * magnitude;
    }
    if (q_gain) {
        sq = ni_block_sum(sq, scratch);
        sk = ni_block_sum(sk, scratch);      // (its barriers also publish row and cs)
    } else {
        __syncthreads();                     // no norm over the whole row: row and cs are all that is needed
    }
    const float inv_q = q_gain ? 1.0f / sqrtf(sq / (float)nq + eps) : 1.0f;
    const float inv_k = k_gain ? 1.0f / sqrtf(sk / (float)nk + eps) : 1.0f;
    T* kdst = nullptr;
    T* vdst = nullptr;
    if (k_pages) {
        const int page = block_table[(size_t)seq_of_token[t] * bt_stride + pos / page_size];
        const int in_page = pos % page_size;
        kdst = k_pages + ((size_t)page * G * page_size + in_page) * D;           // head g: + g * page_size * D
        vdst = v_pages + ((size_t)page * G * page_size + in_page) * V;
    }
    for (int i = threadIdx.x; i < nq + nk; i += blockDim.x) {
        const bool is_q = i < nq;
        const int e = is_q ? i : i - nq;
        const int head = e / D, dim = e - head * D;
        const float* gain = is_q ? q_gain : k_gain;
        const float inv = is_q ? inv_q : inv_k;
        float a = row[i] * inv * (gain ? gain[e] : 1.0f);
        if (dim < rotary_dim) {
            const bool first = dim < half;
            const int other = first ? i + half : i - half, oe = first ? e + half : e - half;
            const float b = row[other] * inv * (gain ? gain[oe] : 1.0f);
            const int f = first ? dim : dim - half;
            a = first ? a * cs[f] - b * cs[half + f] : a * cs[f] + b * cs[half + f];
        }
        if (head_unit) cs[rotary_dim + i] = a;            // kept for the heads' own norms below
        else if (is_q) q_out[(size_t)t * nq + e] = ni_from_float<T>(a * temp);
        else if (kdst) kdst[(size_t)head * page_size * D + dim] = ni_from_float<T>(a);
    }
    if (head_unit) qk_head_unit_write<T>(cs + rotary_dim, eps, temp, q_out + (size_t)t * nq, kdst, H, G, D, page_size);
    if (vdst) {
        for (int i = threadIdx.x; i < nv; i += blockDim.x) {
            const int head = i / V, dim = i - head * V;
            float v = ni_to_float(x[nq + nk + i]) + (bias ? bias[nq + nk + i] : 0.f);
            if (ex.first_v) {
                const float f = ni_to_float(ex.first_v[(size_t)t * ex.first_ld + i]) + (ex.first_bias ? ex.first_bias[i] : 0.f);
                v = (1.0f - ex.lambda) * v + ex.lambda * f;
            }
            vdst[(size_t)head * page_size * V + dim] = ni_from_float<T>(v);
        }
    }
}

// The same with 16 bytes per load and store: a thread owns VEC neighbouring dimensions (8 bfloat16 or 4 floats).
// For sizes whose heads, rotated halves and rows all start on 16 bytes (the launcher checks).
template <typename TI, typename T>
__global__ void __launch_bounds__(256)
qk_norm_rope_vec_kernel(const TI* __restrict__ qkv, int ld, const float* __restrict__ bias,
                        const float* __restrict__ q_gain, const float* __restrict__ k_gain, float eps,
                        const int* __restrict__ positions, const int* __restrict__ seq_of_token,
                        const int* __restrict__ block_table, int bt_stride, const float* __restrict__ inv_freq,
                        float magnitude, T* __restrict__ q_out, T* __restrict__ k_pages, T* __restrict__ v_pages,
                        int H, int G, int D, int V, int rotary_dim, int page_size, int head_unit, const QkExtra<TI> ex) {
    constexpr int VEC = 16 / sizeof(T);
    extern __shared__ __align__(16) float sm[];
    __shared__ float scratch[32];
    const int nq = H * D, nk = G * D, nv = G * V, half = rotary_dim >> 1;
    float* row = sm;                 // [nq + nk]: queries, then keys, bias added
    float* cs = sm + nq + nk;        // [2 half]: m cos, then m sin
    const int t = blockIdx.x;
    const TI* x = qkv + (size_t)t * ld;
    const int pos = positions[t];
    const float temp = qk_temperature(ex.temp_coef, ex.temp_every, pos);
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x * VEC; i < nq + nk; i += blockDim.x * VEC) {
        float v[VEC];
        qk_load<TI, VEC>(x + i, v);
        if (bias) {
#pragma unroll
            for (int k = 0; k < VEC; k += 4) {
                const float4 b4 = *reinterpret_cast<const float4*>(bias + i + k);
                v[k] += b4.x; v[k + 1] += b4.y; v[k + 2] += b4.z; v[k + 3] += b4.w;
            }
        }
        float ss = 0.f;
#pragma unroll
        for (int k = 0; k < VEC; ++k) ss = fmaf(v[k], v[k], ss);
        if (i < nq) sq += ss; else sk += ss;
#pragma unroll
        for (int k = 0; k < VEC; k += 4) *reinterpret_cast<float4*>(row + i + k) = make_float4(v[k], v[k + 1], v[k + 2], v[k + 3]);
    }
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        float s, c;
        sincosf((float)pos * inv_freq[i], &s, &c);
        cs[i] = c * magnitude;
        cs[half + i] = s * magnitude;
    }
    T* kdst = nullptr;
    T* vdst = nullptr;
    if (k_pages) {
        const int page = block_table[(size_t)seq_of_token[t] * bt_stride + pos / page_size];
        const int in_page = pos % page_size;
        kdst = k_pages + ((size_t)page * G * page_size + in_page) * D;           // head g: + g * page_size * D
        vdst = v_pages + ((size_t)page * G * page_size + in_page) * V;
    }
    if (vdst) {                               // the values do not wait for the sums
        for (int i = threadIdx.x * VEC; i < nv; i += blockDim.x * VEC) {
            const int head = i / V, dim = i - head * V;
            float v[VEC];
            qk_load<TI, VEC>(x + nq + nk + i, v);
            if (bias) {
#pragma unroll
                for (int k = 0; k < VEC; ++k) v[k] += bias[nq + nk + i + k];
            }
            if (ex.first_v) {
                float f[VEC];
                qk_load<TI, VEC>(ex.first_v + (size_t)t * ex.first_ld + i, f);
#pragma unroll
                for (int k = 0; k < VEC; ++k)
                    v[k] = (1.0f - ex.lambda) * v[k] + ex.lambda * (f[k] + (ex.first_bias ? ex.first_bias[i + k] : 0.f));
            }
            NiVec16<T>::store(vdst + (size_t)head * page_size * V + dim, v);
        }
    }
    if (q_gain) {
        sq = ni_block_sum(sq, scratch);
        sk = ni_block_sum(sk, scratch);      // (its barriers also publish row and cs)
    } else {
        __syncthreads();                     // no norm over the whole row: row and cs are all that is needed
    }
    const float inv_q = q_gain ? 1.0f / sqrtf(sq / (float)nq + eps) : 1.0f;
    const float inv_k = k_gain ? 1.0f / sqrtf(sk / (float)nk + eps) : 1.0f;
    for (int i = threadIdx.x * VEC; i < nq + nk; i += blockDim.x * VEC) {
        const bool is_q = i < nq;
        const int e = is_q ? i : i - nq;
        const int head = e / D, dim = e - head * D;
        const float* gain = is_q ? q_gain : k_gain;
        const float inv = is_q ? inv_q : inv_k;
        float a[VEC];
#pragma unroll
        for (int k = 0; k < VEC; ++k) a[k] = row[i + k] * inv * (gain ? gain[e + k] : 1.0f);
        if (dim < rotary_dim) {               // all VEC dimensions lie in the same half
            const bool first = dim < half;
            const int shift = first ? half : -half;
            const int f = first ? dim : dim - half;
#pragma unroll
            for (int k = 0; k < VEC; ++k) {
                const float b = row[i + shift + k] * inv * (gain ? gain[e + shift + k] : 1.0f);
                a[k] = first ? a[k] * cs[f + k] - b * cs[half + f + k] : a[k] * cs[f + k] + b * cs[half + f + k];
            }
        }
        if (head_unit) {                       // kept for the heads' own norms below
#pragma unroll
            for (int k = 0; k < VEC; ++k) cs[rotary_dim + i + k] = a[k];
            continue;
        }
        uint4 packed;
        T* o = reinterpret_cast<T*>(&packed);
#pragma unroll
        for (int k = 0; k < VEC; ++k) o[k] = ni_from_float<T>(is_q ? a[k] * temp : a[k]);
        if (is_q) *reinterpret_cast<uint4*>(q_out + (size_t)t * nq + e) = packed;
        else if (kdst) *reinterpret_cast<uint4*>(kdst + (size_t)head * page_size * D + dim) = packed;
    }
    if (head_unit) qk_head_unit_write<T>(cs + rotary_dim, eps, temp, q_out + (size_t)t * nq, kdst, H, G, D, page_size);
}

// Without norms over the whole row, for heads of 64 or 128 that are rotated whole or not at all: a warp per head, the two
// dimensions of a rotated pair in one lane (a lane owns E neighbours of the first half and their partners), the head's own norm
// by shuffles, nothing in shared memory.  Up to four heads per warp are on their way at a time; cosines and sines once per warp.
template <typename TI, int E> __device__ __forceinline__ void qk_load_e(const TI* p, float* v);
template <> __device__ __forceinline__ void qk_load_e<float, 1>(const float* p, float* v) { v[0] = *p; }
template <> __device__ __forceinline__ void qk_load_e<__nv_bfloat16, 1>(const __nv_bfloat16* p, float* v) { v[0] = __bfloat162float(*p); }
template <> __device__ __forceinline__ void qk_load_e<float, 2>(const float* p, float* v) {
    const float2 x = *reinterpret_cast<const float2*>(p);
    v[0] = x.x; v[1] = x.y;
}
template <> __device__ __forceinline__ void qk_load_e<__nv_bfloat16, 2>(const __nv_bfloat16* p, float* v) {
    const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
    v[0] = x.x; v[1] = x.y;
}
__device__ __forceinline__ void qk_store_e(float* p, const float* v, int e) {
    if (e == 1) *p = v[0];
    else *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]);
}
__device__ __forceinline__ void qk_store_e(__nv_bfloat16* p, const float* v, int e) {
    if (e == 1) *p = __float2bfloat16_rn(v[0]);
    else *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v[0], v[1]);
}

template <typename TI, typename T, int E>
__global__ void __launch_bounds__(256)
qk_heads_kernel(const TI* __restrict__ qkv, int ld, const float* __restrict__ bias, float eps, const int* __restrict__ positions,
                const int* __restrict__ seq_of_token, const int* __restrict__ block_table, int bt_stride,
                const float* __restrict__ inv_freq, float magnitude, T* __restrict__ q_out, T* __restrict__ k_pages,
                T* __restrict__ v_pages, int H, int G, int V, int rotated, int page_size, int head_unit,
                const QkExtra<TI> ex) {
    constexpr int D = 64 * E, HALF = 32 * E, VEC = 16 / sizeof(T), AT_ONCE = 4;
    const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    const TI* x = qkv + (size_t)t * ld;
    const int pos = positions[t], nq = H * D, nk = G * D, nv = G * V;
    const float temp = qk_temperature(ex.temp_coef, ex.temp_every, pos);
    T* kdst = nullptr;
    T* vdst = nullptr;
    if (k_pages) {
        const int page = block_table[(size_t)seq_of_token[t] * bt_stride + pos / page_size], in_page = pos % page_size;
        kdst = k_pages + ((size_t)page * G * page_size + in_page) * D;
        vdst = v_pages + ((size_t)page * G * page_size + in_page) * V;
    }
    float cs[E], sn[E];
#pragma unroll
    for (int e = 0; e < E; ++e) {
        cs[e] = 1.f;
        sn[e] = 0.f;
        if (rotated) {
            sincosf((float)pos * inv_freq[E * lane + e], &sn[e], &cs[e]);
            cs[e] *= magnitude;
            sn[e] *= magnitude;
        }
    }
    const int heads = kdst ? H + G : H;
    for (int h0 = warp; h0 < heads; h0 += AT_ONCE * warps) {
        float a[AT_ONCE][E], b[AT_ONCE][E];
#pragma unroll
        for (int k = 0; k < AT_ONCE; ++k) {
            const int head = h0 + k * warps;
            if (head < heads) {
                qk_load_e<TI, E>(x + (size_t)head * D + E * lane, a[k]);
                qk_load_e<TI, E>(x + (size_t)head * D + HALF + E * lane, b[k]);
            }
        }
#pragma unroll
        for (int k = 0; k < AT_ONCE; ++k) {
            const int head = h0 + k * warps;
            if (head >= heads) break;
            float ss = 0.f;
#pragma unroll
            for (int e = 0; e < E; ++e) {
                float u = a[k][e], v = b[k][e];
                if (bias) {
                    u += bias[head * D + E * lane + e];
                    v += bias[head * D + HALF + E * lane + e];
                }
                a[k][e] = u * cs[e] - v * sn[e];
                b[k][e] = v * cs[e] + u * sn[e];
                ss = fmaf(a[k][e], a[k][e], fmaf(b[k][e], b[k][e], ss));
            }
            float f = head < H ? temp : 1.f;
            if (head_unit) f /= sqrtf(ni_warp_sum(ss) / (float)D + eps);
#pragma unroll
            for (int e = 0; e < E; ++e) { a[k][e] *= f; b[k][e] *= f; }
            T* dst = head < H ? q_out + (size_t)t * nq + (size_t)head * D : kdst + (size_t)(head - H) * page_size * D;
            qk_store_e(dst + E * lane, a[k], E);
            qk_store_e(dst + HALF + E * lane, b[k], E);
        }
    }
    if (!vdst) return;
    for (int i = threadIdx.x * VEC; i < nv; i += blockDim.x * VEC) {
        const int head = i / V, dim = i - head * V;
        float v[VEC];
        qk_load<TI, VEC>(x + nq + nk + i, v);
        if (bias) {
#pragma unroll
            for (int k = 0; k < VEC; ++k) v[k] += bias[nq + nk + i + k];
        }
        if (ex.first_v) {
            float f[VEC];
            qk_load<TI, VEC>(ex.first_v + (size_t)t * ex.first_ld + i, f);
#pragma unroll
            for (int k = 0; k < VEC; ++k)
                v[k] = (1.0f - ex.lambda) * v[k] + ex.lambda * (f[k] + (ex.first_bias ? ex.first_bias[i + k] : 0.f));
        }
        NiVec16<T>::store(vdst + (size_t)head * page_size * V + dim, v);
    }
}

// qkv [T, ld] with columns q (H D) | k (G D) | v (G V); bias FP32 [H D + G D + G V] or null; q_gain FP32 [H D] and
// k_gain FP32 [G D], or null for no norm; head_unit: the heads' own norms after the rotation; k_pages / v_pages null: nothing is written (a run that reads another's cache).
// dtype: queries and pages; in_dtype: qkv and first_v (FP32 beside bfloat16 is allowed).  temp_coef 0: no factor on the
// query.  first_v null: no mixing of values; else the other layer's value columns, row stride first_ld (see QkExtra).
NI_EXPORT int ni_qk_norm_rope(const void* qkv, int in_dtype, int dtype, int ld, const float* bias, const float* q_gain,
                              const float* k_gain, float eps, const int* positions, const int* seq_of_token,
                              const int* block_table, int bt_stride, const float* inv_freq, float magnitude, void* q_out,
                              void* k_pages, void* v_pages, int n_tokens, int H, int G, int D, int V, int rotary_dim,
                              int page_size, int head_unit, float temp_coef, float temp_every, const void* first_v,
                              int first_ld, const float* first_bias, float lambda, cudaStream_t stream) {
    if (n_tokens <= 0) return NI_OK;
    if (H <= 0 || G <= 0 || D <= 0 || V <= 0 || page_size <= 0 || rotary_dim < 0 || rotary_dim > D || (rotary_dim & 1) ||
        ld < (H + G) * D + G * V || (q_gain == nullptr) != (k_gain == nullptr) || (first_v && first_ld < G * V) ||
        (temp_coef != 0.f && !(temp_every > 0.f)))
        return NI_ERR_BAD_ARGUMENT;
    const size_t smem = ((size_t)(H + G) * D * (head_unit ? 2 : 1) + rotary_dim) * sizeof(float);
    if (smem > 200 * 1024) return NI_ERR_UNSUPPORTED_SIZE;
    const int vec = dtype == NI_DTYPE_F32 ? 4 : 8;       // elements in 16 bytes of the output
    const auto aligned = [](const void* p) { return (reinterpret_cast<size_t>(p) & 15) == 0; };
    const bool wide = D % vec == 0 && V % vec == 0 && (rotary_dim / 2) % vec == 0 && ld % vec == 0 && aligned(qkv) &&
                      aligned(q_out) && aligned(k_pages) && aligned(v_pages) && aligned(bias) && first_ld % vec == 0 &&
                      aligned(first_v);
    const int work = ((H + G) * D + vec - 1) / vec;
    const int threads = !wide ? 256 : (work >= 256 ? 256 : (work >= 128 ? 128 : 64));
#define LAUNCH_K(KERNEL, TI, T)                                                                                      \
    do {                                                                                                             \
        const QkExtra<TI> ex = {temp_coef, temp_every, (const TI*)first_v, first_ld, first_bias, lambda};            \
        if (smem > 48 * 1024)                                                                                        \
            cudaFuncSetAttribute(KERNEL<TI, T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);             \
        KERNEL<TI, T><<<n_tokens, threads, smem, stream>>>((const TI*)qkv, ld, bias, q_gain, k_gain, eps, positions, \
                                                           seq_of_token, block_table, bt_stride, inv_freq, magnitude, \
                                                           (T*)q_out, (T*)k_pages, (T*)v_pages, H, G, D, V,          \
                                                           rotary_dim, page_size, head_unit, ex);                    \
    } while (0)
#define LAUNCH_H(TI, T, E)                                                                                           \
    do {                                                                                                             \
        const QkExtra<TI> ex = {temp_coef, temp_every, (const TI*)first_v, first_ld, first_bias, lambda};            \
        qk_heads_kernel<TI, T, E><<<n_tokens, 256, 0, stream>>>((const TI*)qkv, ld, bias, eps, positions, seq_of_token, \
                                                                block_table, bt_stride, inv_freq, magnitude, (T*)q_out, \
                                                                (T*)k_pages, (T*)v_pages, H, G, V, rotary_dim > 0,   \
                                                                page_size, head_unit, ex);                           \
    } while (0)
    const bool by_heads = wide && !q_gain && (D == 64 || D == 128) && (rotary_dim == 0 || rotary_dim == D);
#define LAUNCH(TI, T)                                                \
    do {                                                             \
        if (by_heads && D == 64) LAUNCH_H(TI, T, 1);                 \
        else if (by_heads) LAUNCH_H(TI, T, 2);                       \
        else if (wide) LAUNCH_K(qk_norm_rope_vec_kernel, TI, T);          \
        else LAUNCH_K(qk_norm_rope_kernel, TI, T);                   \
    } while (0)
    if (dtype == NI_DTYPE_F32 && in_dtype == NI_DTYPE_F32) LAUNCH(float, float);
    else if (dtype == NI_DTYPE_BF16 && in_dtype == NI_DTYPE_BF16) LAUNCH(__nv_bfloat16, __nv_bfloat16);
    else if (dtype == NI_DTYPE_BF16 && in_dtype == NI_DTYPE_F32) LAUNCH(float, __nv_bfloat16);
    else return NI_ERR_BAD_ARGUMENT;
#undef LAUNCH
#undef LAUNCH_H
#undef LAUNCH_K
    NI_RETURN_LAUNCH_STATUS();
}
