// The difference of two attention maps per head, normed: u = a_1 - lambda a_2, out = u / sqrt(mean(u^2) + eps) * factor.
// a FP32 [T, H, 2, V]; out [T, H, V].  One warp per (token, head); FP32 throughout.
#include "common.cuh"

template <typename T>
__global__ void __launch_bounds__(128)
difference_norm_kernel(const float* __restrict__ a, T* __restrict__ out, const int* __restrict__ token_list, long long items, int H,
                       int V, float lambda, float eps, float factor) {
    const long long item = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
    if (item >= items) return;
    const int lane = threadIdx.x & 31;
    const long long i = item / H;
    const int h = (int)(item - i * H);
    const size_t t = token_list ? token_list[i] : i;
    const float* a1 = a + (t * H + h) * 2 * V;
    const float* a2 = a1 + V;
    float ss = 0.f;
    for (int v = lane; v < V; v += 32) {
        const float u = fmaf(-lambda, a2[v], a1[v]);
        ss = fmaf(u, u, ss);
    }
    ss = ni_warp_sum(ss);
    const float r = factor / sqrtf(ss / (float)V + eps);
    T* o = out + (t * H + h) * V;
    for (int v = lane; v < V; v += 32) o[v] = ni_from_float<T>(fmaf(-lambda, a2[v], a1[v]) * r);
}

NI_EXPORT int ni_difference_norm(const float* a, void* out, int dtype, const int* token_list, int n_tokens, int H, int V, float lambda,
                                 float eps, float factor, cudaStream_t stream) {
    if (n_tokens <= 0) return NI_OK;
    if (H <= 0 || V <= 0) return NI_ERR_BAD_ARGUMENT;
    const long long items = (long long)n_tokens * H, blocks = (items + 3) / 4;
    if (blocks > 2147483647LL) return NI_ERR_UNSUPPORTED_SIZE;
    if (dtype == NI_DTYPE_F32)
        difference_norm_kernel<float><<<(int)blocks, 128, 0, stream>>>(a, (float*)out, token_list, items, H, V, lambda, eps, factor);
    else if (dtype == NI_DTYPE_BF16)
        difference_norm_kernel<__nv_bfloat16><<<(int)blocks, 128, 0, stream>>>(a, (__nv_bfloat16*)out, token_list, items, H, V, lambda, eps, factor);
    else
        return NI_ERR_BAD_ARGUMENT;
    NI_RETURN_LAUNCH_STATUS();
}
