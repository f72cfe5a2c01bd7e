// Causal grouped-query attention over the paged cache, the plain way: one warp per
// (token, query head), keys visited one by one in ascending position with an online
// softmax in FP32.  Prompt portions and single decoded tokens are the same case: a
// token at position p sees keys [max(0, p - window + 1), p] of its own request.  An optional
// token list restricts the launch to some of the step's tokens (n_tokens = its length).
// An optional slope per query head adds slope * (key position - query position) to the scaled
// score: a position encoding that acts on the scores instead of rotating queries and keys.
// An optional cap bounds the scaled score smoothly: s <- cap * tanh(s / cap) (cap = 0: none), FP32, before
// the bias and the softmax.
// Values may have a size of their own (v_dim): the value pages are then [P, Hkv, page, v_dim] and the output
// [T, Hq, v_dim].
// Two more masks and one more denominator, all parameters: `chunk` > 0 lets a token see only the keys of its own
// chunk, [p - p % chunk, p], chunks counted from the sequence's position 0; `sinks` (one number per query head) adds
// exp(sinks[head]) to the softmax's denominator - a key of that score without a value - so the weights of a token sum to
// less than one.
// `maps` > 1: every head has that many attention maps of its own over the same values.  q is then [T, Hq] rows of
// head_dim, Hq counting maps (head h's map m is row h * maps + m), a key row holds the maps side by side (maps * head_dim
// numbers), and every map has an output row of v_dim numbers.  The output may be FP32 whatever the inputs' type.
//
// The result of a token depends only on its own keys and their order, never on how the
// step was cut or what else is in the batch, so this kernel is the FP32 path's attention
// and the yardstick beside the tensor-core kernels.
//
// Formula as in the reference (decode: src/op/kernels/cuda/paged_attention_kernel.cu:124-198,
// prefill: prefill_attention_kernel.cu:66-141): score = (q . k) * scale, softmax with the
// maximum subtracted, out = sum p_j v_j, kv head = q head / (Hq / Hkv).  The reference
// divides by (sum + 1e-6); this kernel divides by the sum.
#include "common.cuh"

// Registers per lane for a head: 8 take head sizes up to 256; a second instance with 16 takes up to 512 and a third
// with 32 up to 1,024 (a compressed cache row can be that wide); each leaves the others as they were.
template <typename T, typename TO, int ATT_MAX_REGS>
__global__ void attention_generic_kernel(const T* __restrict__ q, const T* __restrict__ k_pages,
                                         const T* __restrict__ v_pages, TO* __restrict__ out,
                                         const int* __restrict__ token_list,
                                         const int* __restrict__ positions,
                                         const int* __restrict__ seq_of_token,
                                         const int* __restrict__ block_table, int bt_stride,
                                         int n_tokens, int n_q_heads, int n_kv_heads, int head_dim,
                                         int page_size, int window, float scale,
                                         const float* __restrict__ head_slopes, float score_cap, int v_dim, int chunk,
                                         const float* __restrict__ sinks, int maps) {
    const int warps_per_block = blockDim.x >> 5;
    const long long item = (long long)blockIdx.x * warps_per_block + (threadIdx.x >> 5);
    if (item >= (long long)n_tokens * n_q_heads) return;
    const int lane = threadIdx.x & 31;
    const int t_item = (int)(item / n_q_heads);
    const int head = (int)(item - (long long)t_item * n_q_heads);
    const int t = token_list ? token_list[t_item] : t_item;
    const int kvh = head / (n_q_heads / n_kv_heads);
    const int pos = positions[t];
    const int* table = block_table + (size_t)seq_of_token[t] * bt_stride;
    int lo = (window > 0 && pos - window + 1 > 0) ? pos - window + 1 : 0;
    if (chunk > 0 && pos - pos % chunk > lo) lo = pos - pos % chunk;
    const float slope = head_slopes ? head_slopes[head] : 0.f;
    const int k_row = maps * head_dim, k_off = (head % maps) * head_dim;

    float qr[ATT_MAX_REGS], acc[ATT_MAX_REGS];
    const T* qrow = q + ((size_t)t * n_q_heads + head) * head_dim;
#pragma unroll
    for (int r = 0; r < ATT_MAX_REGS; ++r) {
        const int dim = lane + 32 * r;
        qr[r] = dim < head_dim ? ni_to_float(qrow[dim]) : 0.f;
        acc[r] = 0.f;
    }
    float m = sinks ? sinks[head] : -INFINITY, l = sinks ? 1.f : 0.f;      // the sink: a key that is there from the start
    for (int j = lo; j <= pos; ++j) {
        const int page = table[j / page_size];
        const size_t slot = ((size_t)page * n_kv_heads + kvh) * page_size + (j % page_size);
        const T* krow = k_pages + slot * k_row + k_off;
        const T* vrow = v_pages + slot * v_dim;
        float dot = 0.f;
#pragma unroll
        for (int r = 0; r < ATT_MAX_REGS; ++r) {
            const int dim = lane + 32 * r;
            if (dim < head_dim) dot += qr[r] * ni_to_float(krow[dim]);
        }
        dot = ni_warp_sum(dot);
        float s = dot * scale;
        if (score_cap > 0.f) s = score_cap * tanhf(s / score_cap);
        s += slope * (float)(j - pos);
        const float m_new = fmaxf(m, s);
        const float corr = expf(m - m_new);  // exp(-inf) = 0 on the first key
        const float p = expf(s - m_new);
        l = l * corr + p;
#pragma unroll
        for (int r = 0; r < ATT_MAX_REGS; ++r) {
            const int dim = lane + 32 * r;
            if (dim < v_dim) acc[r] = acc[r] * corr + p * ni_to_float(vrow[dim]);
        }
        m = m_new;
    }
    TO* orow = out + ((size_t)t * n_q_heads + head) * v_dim;
    const float inv = 1.0f / l;
#pragma unroll
    for (int r = 0; r < ATT_MAX_REGS; ++r) {
        const int dim = lane + 32 * r;
        if (dim < v_dim) orow[dim] = ni_from_float<TO>(acc[r] * inv);
    }
}

NI_EXPORT int ni_attention_generic(const void* q, int dtype, const void* k_pages,
                                   const void* v_pages, void* out, int out_dtype, const int* token_list,
                                   const int* positions, const int* seq_of_token, const int* block_table, int bt_stride,
                                   int n_tokens, int n_q_heads, int n_kv_heads, int head_dim,
                                   int page_size, int window, float scale, const float* head_slopes,
                                   float score_cap, int v_dim, int chunk, const float* sinks, int maps, cudaStream_t stream) {
    if (n_tokens <= 0) return NI_OK;
    if (n_q_heads <= 0 || n_kv_heads <= 0 || n_q_heads % n_kv_heads || head_dim <= 0 || page_size <= 0 || v_dim < 0 || chunk < 0 ||
        maps <= 0 || (n_q_heads / n_kv_heads) % maps)
        return NI_ERR_BAD_ARGUMENT;
    if (v_dim == 0) v_dim = head_dim;          // values of the keys' size
    if (head_dim > 32 * 32 || v_dim > 32 * 32) return NI_ERR_UNSUPPORTED_SIZE;
    const int warps = 4;
    const long long items = (long long)n_tokens * n_q_heads;
    const long long blocks = (items + warps - 1) / warps;
    if (blocks > 2147483647LL) return NI_ERR_UNSUPPORTED_SIZE;
#define LAUNCH_R(T, TO, R)                                                                          \
    attention_generic_kernel<T, TO, R><<<(int)blocks, warps * 32, 0, stream>>>(                     \
        (const T*)q, (const T*)k_pages, (const T*)v_pages, (TO*)out, token_list, positions,        \
        seq_of_token,                                                                               \
        block_table, bt_stride, n_tokens, n_q_heads, n_kv_heads, head_dim, page_size, window, scale, head_slopes, score_cap, v_dim, chunk, sinks, maps)
#define LAUNCH(T, TO)                      \
    do {                                   \
        if (head_dim <= 256 && v_dim <= 256) LAUNCH_R(T, TO, 8); \
        else if (head_dim <= 512 && v_dim <= 512) LAUNCH_R(T, TO, 16); \
        else LAUNCH_R(T, TO, 32);              \
    } while (0)
    if (dtype == NI_DTYPE_F32 && out_dtype == NI_DTYPE_F32) LAUNCH(float, float);
    else if (dtype == NI_DTYPE_BF16 && out_dtype == NI_DTYPE_BF16) LAUNCH(__nv_bfloat16, __nv_bfloat16);
    else if (dtype == NI_DTYPE_BF16 && out_dtype == NI_DTYPE_F32) LAUNCH(__nv_bfloat16, float);
    else return NI_ERR_BAD_ARGUMENT;
#undef LAUNCH
#undef LAUNCH_R
    NI_RETURN_LAUNCH_STATUS();
}
