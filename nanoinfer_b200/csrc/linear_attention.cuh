// What the chunked linear-attention kernels share (lightning attention, retention, matrix memories): chunks of LT_C tokens,
// tile loads into shared memory, the place of a request's chunks in the step's buffer, and the warp-level pieces of the
// tensor-core variants (mma.sync with bfloat16 operands, transposing shared-memory loads, splitting an FP32 number into
// two bfloat16 halves, asynchronous copies).
#pragma once
#include "common.cuh"

#define LT_C 64          // tokens per chunk
#define LT_THREADS 256
#define LT_KV_TILE 64    // rows and columns of a chunk's sum that one block of lightning_chunk_kv_kernel owns

__device__ __forceinline__ float lt_silu(float z) { return z / (1.0f + expf(-z)); }
// The activation of a projection's entry, in the projection's own type: bfloat16 projections give the bfloat16 rounding
// of silu, in every kernel of this file alike, so that a prompt's portion and single tokens read the same q, k and v.
template <typename T> __device__ __forceinline__ float lt_act(T raw) { return ni_to_float(ni_from_float<T>(lt_silu(ni_to_float(raw)))); }
// The fast exponential and division are exact enough for a result that is rounded to 8 bits of mantissa.
template <> __device__ __forceinline__ float lt_act<__nv_bfloat16>(__nv_bfloat16 raw) {
    const float z = __bfloat162float(raw);
    return __bfloat162float(__float2bfloat16_rn(__fdividef(z, 1.0f + __expf(-z))));
}

// An FP32 entry that enters the recurrence as it is (no activation): the caller has made q, k and v itself, for
// instance rotated queries and scaled keys of a retention layer.  A type of its own, so that the FP32 FMA kernels
// below get a second instance and the ones with silu stay as they are.
struct LtPlain { float v; };
template <> __device__ __forceinline__ float ni_to_float<LtPlain>(LtPlain x) { return x.v; }
template <> __device__ __forceinline__ float lt_act<LtPlain>(LtPlain raw) { return raw.v; }

// dst[r * dst_stride + c] = f(src[r * ld + c]) * scale[r] for r < rows, c < cols (zero for rows .. rows_pad - 1 and
// c in cols .. cols_pad - 1).  16 bytes per load when every row starts on 16 bytes and cols is a multiple of the
// vector's elements.
template <typename T, bool SILU>
__device__ __forceinline__ void lt_load_tile(const T* __restrict__ src, size_t ld, int rows, int rows_pad, int cols, int cols_pad,
                                             float* __restrict__ dst, int dst_stride, const float* __restrict__ row_scale,
                                             int scale_last) {
    constexpr int VEC = 16 / sizeof(T);
    const bool wide = cols % VEC == 0 && ld % VEC == 0 && (reinterpret_cast<size_t>(src) & 15) == 0 && cols_pad % 4 == 0 &&
                      dst_stride % 4 == 0;
    if (wide) {
        const int per_row = cols_pad / VEC + (cols_pad % VEC ? 1 : 0);
        for (int i = threadIdx.x; i < rows_pad * per_row; i += LT_THREADS) {
            const int r = i / per_row, c = (i - r * per_row) * VEC;
            float v[VEC];
            if (r < rows && c < cols) {
                const uint4 raw = *reinterpret_cast<const uint4*>(src + (size_t)r * ld + c);
                const T* e = reinterpret_cast<const T*>(&raw);
                const float sc = row_scale ? row_scale[scale_last - r] : 1.0f;
#pragma unroll
                for (int k = 0; k < VEC; ++k) {
                    v[k] = (SILU ? lt_act<T>(e[k]) : ni_to_float(e[k])) * sc;
                }
            } else {
#pragma unroll
                for (int k = 0; k < VEC; ++k) v[k] = 0.f;
            }
#pragma unroll
            for (int k = 0; k < VEC; k += 4)
                if (c + k < cols_pad)
                    *reinterpret_cast<float4*>(dst + r * dst_stride + c + k) = make_float4(v[k], v[k + 1], v[k + 2], v[k + 3]);
        }
        return;
    }
    for (int i = threadIdx.x; i < rows_pad * cols_pad; i += LT_THREADS) {
        const int r = i / cols_pad, c = i - r * cols_pad;
        float v = 0.f;
        if (r < rows && c < cols) {
            const T raw = src[(size_t)r * ld + c];
            v = (SILU ? lt_act<T>(raw) : ni_to_float(raw)) * (row_scale ? row_scale[scale_last - r] : 1.0f);
        }
        dst[r * dst_stride + c] = v;
    }
}

// The first chunk of request `seq` in the buffer: the chunks of the requests before it, counted by all threads.
__device__ __forceinline__ int lt_chunk_base(const int* __restrict__ cu_q, int seq, int* scratch) {
    if (threadIdx.x == 0) *scratch = 0;
    __syncthreads();
    int mine = 0;
    for (int s = threadIdx.x; s < seq; s += blockDim.x) mine += (cu_q[s + 1] - cu_q[s] + LT_C - 1) / LT_C;
    if (mine) atomicAdd(scratch, mine);
    __syncthreads();
    return *scratch;
}

__device__ __forceinline__ void lt_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Four 8 x 8 blocks of 16-bit numbers, each transposed on the way: lane l gives the address of row l % 8 of block l / 8.
__device__ __forceinline__ void lt_ldsm_x4_trans(uint32_t (&r)[4], const void* p) {
    const uint32_t addr = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void lt_split2(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const float2 hf = __bfloat1622float2(h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - hf.x, y - hf.y);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ void lt_cp_async16(void* smem, const void* gmem) {
    const uint32_t addr = (uint32_t)__cvta_generic_to_shared(smem);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(addr), "l"(gmem));
}
__device__ __forceinline__ void lt_cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
// Waits until at most N of the thread's committed groups are still under way.
template <int N> __device__ __forceinline__ void lt_cp_async_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N) : "memory"); }
// Rows [0, rows) x columns [0, cols) of src copied as they are (asynchronously, 16 bytes a piece) into dst, zeros up to
// rows_pad x cols_pad; lt_activate_own then turns the pieces that the same thread copied into their activations, in place
// (times scale[scale_last - r], the remainder of the rounding into dst_lo if given).
// Calls piece(r, c) for every 8-number piece (row r, first column c) of rows x cols_pad, thread by thread; the same thread
// gets the same pieces in every call with the same sizes.  When a row's pieces divide the block, a thread keeps its
// column and steps down the rows (no division per piece).
template <int THREADS, typename F>
__device__ __forceinline__ void lt_for_pieces(int rows, int cols_pad, F piece) {
    const int per_row = cols_pad / 8;
    if (THREADS % per_row == 0) {
        const int c = (threadIdx.x % per_row) * 8, dr = THREADS / per_row;
#pragma unroll 4
        for (int r = threadIdx.x / per_row; r < rows; r += dr) piece(r, c);
    } else {
        for (int i = threadIdx.x; i < rows * per_row; i += THREADS) piece(i / per_row, (i % per_row) * 8);
    }
}
template <int THREADS>
__device__ __forceinline__ void lt_copy_raw(const __nv_bfloat16* __restrict__ src, size_t ld, int rows, int rows_pad, int cols,
                                            int cols_pad, __nv_bfloat16* __restrict__ dst, int dst_stride) {
    lt_for_pieces<THREADS>(rows_pad, cols_pad, [&](int r, int c) {
        if (r < rows && c < cols) lt_cp_async16(dst + r * dst_stride + c, src + (size_t)r * ld + c);
        else *reinterpret_cast<uint4*>(dst + r * dst_stride + c) = make_uint4(0u, 0u, 0u, 0u);
    });
}
