// The gated delta rule with decays per key channel over prompt portions, in chunks of DC_C tokens: matrix products on tensor
// cores instead of a chain of rank-one updates.  For bfloat16 models; the numbers of the recurrence are FP32 throughout - what
// a tensor-core product has to read of them is split into two bfloat16 halves (three products: high x high, low x high, high x
// low), with FP32 accumulation.  (delta_rule.cu runs the same recurrence token by token.)
//
// Per head, with S [D, V] before the chunk, g_i the decays of token i (a number per row of S) and P_i their products up to
// and including token i:
//     u_i = beta_i (v_i - S^T (P_i k_i) - sum_{s<i} A_is u_s)        A_is = sum_d k_i k_s (g_{s+1} .. g_i)
//     o_i = S^T (P_i q_i) + sum_{s<=i} B_is u_s                       B_is = sum_d q_i k_s (g_{s+1} .. g_i)
//     S  <- P_n S + sum_s (k_s g_{s+1} .. g_n) u_s^T
// Only products of decays over a stretch of tokens appear, never their quotients, so nothing overflows however fast a
// channel decays.  The sum over s < i is resolved once per chunk: u = U0 - W S with U0 and W the forward substitutions of
// beta v and beta P k.
//
// Two launches, from the projection (bfloat16) on; the projection's q, k and v never exist in FP32 in memory:
//   delta_chunk_prepare   per (chunk, head), all at once: convolution and silu of the head's channels (a thread per channel
//                         walks the tokens), unit norms, decays, beta - all into shared memory -; A, B (a group of 8 lanes
//                         per s walks i upwards with k_s times the decays in registers - what is left at the end is the
//                         last line's factor); then a thread per column of [W | U0] does the substitution
//   delta_chunk_scan      per (request, head, 16 value columns): the chunks one after the other; S stands in the
//                         accumulators of its warps, and as two bfloat16 planes in shared memory for the products that
//                         read it; the operands of the next two chunks are on their way (bulk copies) while this one's
//                         are used
// The convolution's history is read here and moved on by the gated norm's launch (delta_rule.cu), which follows.
// A chunk begins at a portion's first token, so where a prompt is cut changes results by roundings only.
#include "linear_attention.cuh"

#define DC_C 32          // tokens per chunk
#define DC_THREADS 256
#define DC_VS 16         // value columns per block of the scan
#define DC_AS 36         // row stride of A in shared memory
#define DC_BS (DC_C + 8) // row stride of the planes of B

#define DC_STAGES 3      // chunks whose operands the scan has in shared memory or on their way
#define DC_PAD 8         // numbers behind every row of the planes of W, Q and K (rows then start in different banks)

// One (chunk, head) of the buffer, in bytes - laid out as the scan keeps it in shared memory, so that it is copied as it is: W,
// Q, K as two bfloat16 planes each [DC_C][DP + DC_PAD], the two planes of B [DC_C][DC_BS], P_n FP32 [DP]; behind that U0 FP32
// in slices of DC_VS columns [VP / DC_VS][DC_C][DC_VS].
struct DcLayout {
    int DP, VP;
    __host__ __device__ int rs() const { return DP + DC_PAD; }
    __host__ __device__ size_t plane() const { return (size_t)DC_C * rs() * 2; }
    __host__ __device__ size_t b_off() const { return 6 * plane(); }
    __host__ __device__ size_t p_off() const { return b_off() + 2 * DC_C * DC_BS * 2; }
    __host__ __device__ size_t u_off() const { return p_off() + (size_t)DP * 4; }
    __host__ __device__ size_t bytes() const { return u_off() + (size_t)DC_C * VP * 4; }
};
static int dc_pad_dim(int D) { return D <= 32 ? 32 : (D <= 64 ? 64 : 128); }

// The first chunk of request `seq` in the buffer (called by all threads of the block).
__device__ __forceinline__ int dc_chunk_base(const int* __restrict__ cu_q, int seq, int* scratch) {
    if (threadIdx.x == 0) *scratch = 0;
    __syncthreads();
    int mine = 0;
    for (int s = threadIdx.x; s < seq; s += blockDim.x) mine += (cu_q[s + 1] - cu_q[s] + DC_C - 1) / DC_C;
    if (mine) atomicAdd(scratch, mine);
    __syncthreads();
    return *scratch;
}

__device__ __forceinline__ void dc_store_split(__nv_bfloat16* hi, __nv_bfloat16* lo, float v) {
    const __nv_bfloat16 h = __float2bfloat16_rn(v);
    *hi = h;
    *lo = __float2bfloat16_rn(v - __bfloat162float(h));
}

// What the preparation reads: proj bfloat16 [T, ld] with q (G D) | k (G D) | v (H V) from column 0, beta's logits at b_off;
// z FP32 [T, ld_z], the decays' logits in its first H D columns; a request's convolution history behind its S in state.
struct DcInput {
    const __nv_bfloat16* proj;
    const float *conv_w, *a_log, *dt_bias, *z, *state;
    long long state_stride;
    const int *cu_q, *slots;
    int ld, b_off, ld_z, G, H, D, V, taps;
};

__device__ __forceinline__ float dc_silu(float x) { return __fdividef(x, 1.0f + __expf(-x)); }

// Channel c (of the projection) of the chunk's tokens `first` .. `first + n - 1` through the convolution and silu, rows n ..
// DC_C - 1 zero: dst[r * stride].  TAPS: 4, or 0 for any number.
template <int TAPS>
__device__ __forceinline__ void dc_conv_column(const DcInput& in, const float* __restrict__ hist, int seq_first, int first, int n,
                                               int c, float* dst, int stride) {
    const int taps = TAPS ? TAPS : in.taps, C = 2 * in.G * in.D + in.H * in.V;
    const __nv_bfloat16* x = in.proj + (size_t)first * in.ld + c;
    const int before = first - seq_first;           // tokens of this portion before the chunk
    // the input `back` tokens before the chunk's first: from the portion, or from the history
    const auto earlier = [&](int back) {
        return back <= before ? __bfloat162float(x[-(long long)back * in.ld]) : hist[(size_t)(taps - 1 - (back - before)) * C + c];
    };
    if (TAPS == 4) {
        const float4 w = *reinterpret_cast<const float4*>(in.conv_w + (size_t)c * 4);
        float x3 = earlier(3), x2 = earlier(2), x1 = earlier(1);
        __nv_bfloat16 v[DC_C];
#pragma unroll
        for (int r = 0; r < DC_C; ++r) v[r] = r < n ? x[(size_t)r * in.ld] : __float2bfloat16_rn(0.f);
#pragma unroll
        for (int r = 0; r < DC_C; ++r) {
            const float x0 = __bfloat162float(v[r]);
            const float y = fmaf(w.w, x0, fmaf(w.z, x1, fmaf(w.y, x2, w.x * x3)));
            x3 = x2; x2 = x1; x1 = x0;
            dst[r * stride] = r < n ? dc_silu(y) : 0.f;
        }
    } else {
        for (int r = 0; r < DC_C; ++r) {
            float y = 0.f;
            if (r < n)
                for (int j = 0; j < taps; ++j) {
                    const int back = taps - 1 - j;
                    const float v = back <= r ? __bfloat162float(x[(size_t)(r - back) * in.ld]) : earlier(back - r);
                    y = fmaf(in.conv_w[(size_t)c * taps + j], v, y);
                }
            dst[r * stride] = r < n ? dc_silu(y) : 0.f;
        }
    }
}

// grid (chunks of the longest portion, H, requests).  DP: the padded key size; a lane of the pairs' phase owns DP / 32 groups
// of four channels.
template <int DP, int TAPS>
__global__ void __launch_bounds__(DC_THREADS, 3)
delta_chunk_prepare_kernel(const DcInput in, unsigned char* __restrict__ buf, DcLayout lay) {
    constexpr int M = DP / 32, RS = DP + DC_PAD;
    extern __shared__ __align__(16) float dc_smem[];
    float* sq = dc_smem;                       // [DC_C][DP]
    float* sk = sq + DC_C * DP;
    float* sg = sk + DC_C * DP;
    float* sA = sg + DC_C * DP;                // [DC_C][DC_AS], times beta of the row
    float* sB = sA + DC_C * DC_AS;             // [DC_C][DC_AS]
    float* sv = sB + DC_C * DC_AS;             // [DC_C][VP]
    __shared__ float beta[DC_C];
    __shared__ int base_scratch;
    const int seq = blockIdx.z, h = blockIdx.y;
    const int seq_first = in.cu_q[seq], first = seq_first + blockIdx.x * DC_C, last = in.cu_q[seq + 1];
    if (first >= last) return;
    const int n = min(DC_C, last - first);
    const int H = in.H, G = in.G, D = in.D, V = in.V, VP = lay.VP, g = h / (H / G);
    unsigned char* rec = buf + ((size_t)(dc_chunk_base(in.cu_q, seq, &base_scratch) + blockIdx.x) * H + h) * lay.bytes();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const float* hist = in.state + (size_t)in.slots[seq] * in.state_stride + (size_t)H * D * V;
    // ---- the decays' logits on their way; q, k, v of the chunk; decays; beta ----
    const float* zrow = in.z + (size_t)first * in.ld_z + h * D;
    const bool wide = D % 4 == 0 && in.ld_z % 4 == 0 && (reinterpret_cast<size_t>(in.z) & 15) == 0;
    if (wide) {
        for (int i = tid; i < DC_C * (DP / 4); i += DC_THREADS) {
            const int r = i / (DP / 4), d = 4 * (i % (DP / 4));
            if (r < n && d < D) lt_cp_async16(sg + r * DP + d, zrow + (size_t)r * in.ld_z + d);
        }
    }
    lt_cp_async_commit();
    for (int i = tid; i < 2 * DP + VP; i += DC_THREADS) {
        const int part = i < DP ? 0 : (i < 2 * DP ? 1 : 2), e = i - part * DP;
        float* dst = part == 0 ? sq + e : (part == 1 ? sk + e : sv + e);
        const int stride = part == 2 ? VP : DP;
        if (e < (part == 2 ? V : D)) {
            dc_conv_column<TAPS>(in, hist, seq_first, first, n, part == 2 ? 2 * G * D + h * V + e : part * G * D + g * D + e, dst, stride);
        } else {
            for (int r = 0; r < DC_C; ++r) dst[r * stride] = 0.f;
        }
    }
    lt_cp_async_wait<0>();
    {
        // a thread turns the pieces it copied itself into decays (or fetches number by number where rows are not aligned)
        const float ea = -expf(in.a_log[h]);
        for (int i = tid; i < DC_C * (DP / 4); i += DC_THREADS) {
            const int r = i / (DP / 4), d = 4 * (i % (DP / 4));
            float4* at = reinterpret_cast<float4*>(sg + r * DP + d);
            float4 z4 = *at;
            float* v = reinterpret_cast<float*>(&z4);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const bool live = r < n && d + e < D;
                const float raw = wide ? v[e] : (live ? zrow[(size_t)r * in.ld_z + d + e] : 0.f);
                const float x = live ? raw + in.dt_bias[h * D + d + e] : 0.f;
                v[e] = live ? expf(ea * (x > 20.0f ? x : log1pf(expf(x)))) : 1.f;
            }
            *at = z4;
        }
    }
    for (int i = tid; i < 2 * DC_C * DC_AS; i += DC_THREADS) sA[i] = 0.f;       // A and B
    if (tid < DC_C)
        beta[tid] = tid < n ? 1.0f / (1.0f + expf(-__bfloat162float(in.proj[(size_t)(first + tid) * in.ld + in.b_off + h]))) : 0.f;
    __syncthreads();
    // ---- unit norms: a warp per row ----
    for (int r = warp; r < 2 * DC_C; r += DC_THREADS / 32) {
        float4* row = reinterpret_cast<float4*>((r < DC_C ? sq : sk) + (r & (DC_C - 1)) * DP);
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (lane < DP / 4) v = row[lane];
        const float ss = ni_warp_sum(v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w);
        const float f = 1.0f / sqrtf(ss + 1e-6f) * (r < DC_C ? 1.0f / sqrtf((float)D) : 1.0f);
        if (lane < DP / 4) row[lane] = make_float4(v.x * f, v.y * f, v.z * f, v.w * f);
    }
    __syncthreads();
    {
        // warp w: the tokens s = w, 15 - w, 16 + w, 31 - w (early and late ones together); 8 lanes each.  Four i at a time;
        // their eight sums over the 8 lanes end up one per lane (seven shuffles).
        const int q4 = lane >> 3, l = lane & 7;
        const int s = q4 == 0 ? warp : (q4 == 1 ? 15 - warp : (q4 == 2 ? 16 + warp : 31 - warp));
        float kp[4 * M];
#pragma unroll
        for (int m = 0; m < M; ++m) {
            const float4 v = *reinterpret_cast<const float4*>(sk + s * DP + 4 * (l + 8 * m));
            kp[4 * m] = v.x; kp[4 * m + 1] = v.y; kp[4 * m + 2] = v.z; kp[4 * m + 3] = v.w;
        }
        for (int i0 = warp & ~3; i0 < DC_C; i0 += 4) {
            float t[8];
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const int i = i0 + u;
                const bool decays = i > s;
                float a = 0.f, b = 0.f;
#pragma unroll
                for (int m = 0; m < M; ++m) {
                    const int c = 4 * (l + 8 * m);
                    const float4 gg = *reinterpret_cast<const float4*>(sg + i * DP + c);
                    const float4 kk = *reinterpret_cast<const float4*>(sk + i * DP + c);
                    const float4 qq = *reinterpret_cast<const float4*>(sq + i * DP + c);
                    kp[4 * m] *= decays ? gg.x : 1.f; kp[4 * m + 1] *= decays ? gg.y : 1.f;
                    kp[4 * m + 2] *= decays ? gg.z : 1.f; kp[4 * m + 3] *= decays ? gg.w : 1.f;
                    a = fmaf(kk.x, kp[4 * m], a); a = fmaf(kk.y, kp[4 * m + 1], a);
                    a = fmaf(kk.z, kp[4 * m + 2], a); a = fmaf(kk.w, kp[4 * m + 3], a);
                    b = fmaf(qq.x, kp[4 * m], b); b = fmaf(qq.y, kp[4 * m + 1], b);
                    b = fmaf(qq.z, kp[4 * m + 2], b); b = fmaf(qq.w, kp[4 * m + 3], b);
                }
                t[u] = a;
                t[4 + u] = b;
            }
#pragma unroll
            for (int half = 4; half > 0; half >>= 1) {
                const bool upper = l & half;
#pragma unroll
                for (int e = 0; e < half; ++e) {
                    const float mine = upper ? t[e + half] : t[e], send = upper ? t[e] : t[e + half];
                    t[e] = mine + __shfl_xor_sync(0xffffffffu, send, half);
                }
            }
            const int i = i0 + (l & 3);              // lane l holds the sum of t[l]: A of i0 + l, or B of i0 + l - 4
            if (l < 4 && i > s) sA[i * DC_AS + s] = t[0] * beta[i];
            if (l >= 4 && i >= s) sB[i * DC_AS + s] = t[0];
        }
        __nv_bfloat16* k_hi = reinterpret_cast<__nv_bfloat16*>(rec + 4 * lay.plane()) + s * RS;
        __nv_bfloat16* k_lo = k_hi + DC_C * RS;
#pragma unroll
        for (int m = 0; m < M; ++m) {
            uint2 hi, lo;
            lt_split2(kp[4 * m], kp[4 * m + 1], hi.x, lo.x);
            lt_split2(kp[4 * m + 2], kp[4 * m + 3], hi.y, lo.y);
            *reinterpret_cast<uint2*>(k_hi + 4 * (l + 8 * m)) = hi;
            *reinterpret_cast<uint2*>(k_lo + 4 * (l + 8 * m)) = lo;
        }
    }
    __syncthreads();
    {
        __nv_bfloat16* b_hi = reinterpret_cast<__nv_bfloat16*>(rec + lay.b_off());
        for (int i = tid; i < DC_C * DC_C / 2; i += DC_THREADS) {
            const float2 v = *reinterpret_cast<const float2*>(sB + (i / (DC_C / 2)) * DC_AS + 2 * (i % (DC_C / 2)));
            uint32_t hi, lo;
            lt_split2(v.x, v.y, hi, lo);
            __nv_bfloat16* to = b_hi + (i / (DC_C / 2)) * DC_BS + 2 * (i % (DC_C / 2));
            *reinterpret_cast<uint32_t*>(to) = hi;
            *reinterpret_cast<uint32_t*>(to + DC_C * DC_BS) = lo;
        }
    }
    __nv_bfloat16* w_hi = reinterpret_cast<__nv_bfloat16*>(rec);
    __nv_bfloat16* w_lo = w_hi + DC_C * RS;
    __nv_bfloat16* q_hi = w_lo + DC_C * RS;
    __nv_bfloat16* q_lo = q_hi + DC_C * RS;
    for (int col = tid; col < DP + VP; col += DC_THREADS) {
        const bool is_k = col < DP;
        const int vc = col - DP;
        float* u0 = reinterpret_cast<float*>(rec + lay.u_off()) + (size_t)(vc / DC_VS) * DC_C * DC_VS + vc % DC_VS;
        float x[DC_C], P = 1.f;
#pragma unroll
        for (int i = 0; i < DC_C; ++i) {
            float rhs;
            if (is_k) {
                P *= sg[i * DP + col];
                rhs = sk[i * DP + col] * P;
                dc_store_split(q_hi + i * RS + col, q_lo + i * RS + col, sq[i * DP + col] * P);
            } else {
                rhs = sv[i * VP + vc];
            }
            float acc[4] = {beta[i] * rhs, 0.f, 0.f, 0.f};
#pragma unroll
            for (int s = 0; s < i; s += 4) {
                const float4 a = *reinterpret_cast<const float4*>(sA + i * DC_AS + s);      // zero from column i on
                acc[0] = fmaf(-a.x, x[s], acc[0]);
                if (s + 1 < i) acc[1] = fmaf(-a.y, x[s + 1], acc[1]);
                if (s + 2 < i) acc[2] = fmaf(-a.z, x[s + 2], acc[2]);
                if (s + 3 < i) acc[3] = fmaf(-a.w, x[s + 3], acc[3]);
            }
            x[i] = (acc[0] + acc[1]) + (acc[2] + acc[3]);
            if (is_k) dc_store_split(w_hi + i * RS + col, w_lo + i * RS + col, x[i]);
            else u0[i * DC_VS] = x[i];
        }
        if (is_k) reinterpret_cast<float*>(rec + lay.p_off())[col] = P;
    }
}

__device__ __forceinline__ void dc_ldsm_x4(uint32_t (&r)[4], const void* p) {
    const uint32_t addr = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}

// Bulk copies of whole records into shared memory, counted in by an mbarrier per stage.  A wait lasts at most dc_wait_limit
// clock ticks (about a second); then the error word is set and the kernel returns.  dc_extra_wait: wait once more at the end,
// for a phase that nothing completes (for the test of the give-up path).  Both set by ni_delta_chunk_set_wait.
#define DC_ERR_WAIT 41
__constant__ long long dc_wait_limit = 2000000000LL;
__constant__ int dc_extra_wait = 0;

__device__ __forceinline__ uint32_t dc_smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ bool dc_wait(uint64_t* bar, uint32_t parity, int* error) {
    const uint32_t addr = dc_smem_addr(bar);
    long long start = 0;
    for (int iter = 0;; ++iter) {
        uint32_t done;
        asm volatile(
            "{\n.reg .pred p;\n"
            "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n"
            "selp.b32 %0, 1, 0, p;\n}\n"
            : "=r"(done) : "r"(addr), "r"(parity) : "memory");
        if (done) return true;
        if ((iter & 1023) == 1023) {
            const long long now = clock64();
            if (start == 0) start = now;
            if (now - start > dc_wait_limit) {
                atomicExch(error, DC_ERR_WAIT);
                return false;
            }
        }
    }
}
__device__ __forceinline__ void dc_bulk_copy(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];\n"
                 ::"r"(dc_smem_addr(dst)), "l"(src), "r"(bytes), "r"(dc_smem_addr(bar)) : "memory");
}

template <int DP> __host__ __device__ constexpr int dc_stage_bytes() {
    return 6 * DC_C * (DP + DC_PAD) * 2 + 2 * DC_C * DC_BS * 2 + DP * 4 + DC_C * DC_VS * 4;
}
#define DC_SS (DC_VS + 8)          // row stride of the planes of S and of u
template <int DP> __host__ __device__ constexpr int dc_scan_smem() { return DC_STAGES * dc_stage_bytes<DP>() + 2 * DP * DC_SS * 2 + 2 * DC_C * DC_SS * 2; }

// grid (value slices, H, requests); 8 warps: warp w multiplies row tile w % 4 of [W; Q] with column tile w / 4 of S, and owns
// rows 16 w .. 16 w + 15 of S itself.
template <int DP>
__global__ void __launch_bounds__(DC_THREADS)
delta_chunk_scan_kernel(const unsigned char* __restrict__ buf, DcLayout lay, float* __restrict__ state, long long state_stride,
                        const int* __restrict__ cu_q, const int* __restrict__ slots, int H, int D, int V,
                        float* __restrict__ out, int* __restrict__ error) {
    constexpr int RS = DP + DC_PAD;                  // row stride of the operand planes
    constexpr int FIXED = dc_stage_bytes<DP>() - DC_C * DC_VS * 4;      // of a stage: everything but the slice of U0
    extern __shared__ __align__(16) unsigned char dc_raw[];
    __shared__ int base_scratch;
    const int seq = blockIdx.z, h = blockIdx.y, v0 = blockIdx.x * DC_VS;
    const int first = cu_q[seq], last = cu_q[seq + 1];
    if (first >= last) return;
    const int n_chunks = (last - first + DC_C - 1) / DC_C;
    const unsigned char* rec0 = buf + ((size_t)dc_chunk_base(cu_q, seq, &base_scratch) * H + h) * lay.bytes();
    const size_t rec_step = (size_t)H * lay.bytes();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    __nv_bfloat16* s_hi = reinterpret_cast<__nv_bfloat16*>(dc_raw + DC_STAGES * dc_stage_bytes<DP>());     // [DP][DC_SS]
    __nv_bfloat16* s_lo = s_hi + DP * DC_SS;
    __nv_bfloat16* u_hi = s_lo + DP * DC_SS;                                                         // [DC_C][DC_SS]
    __nv_bfloat16* u_lo = u_hi + DC_C * DC_SS;
    float* S = state + (size_t)slots[seq] * state_stride + (size_t)h * D * V;

    __shared__ __align__(8) uint64_t full[DC_STAGES];
    if (tid == 0) {
        for (int i = 0; i < DC_STAGES; ++i)
            asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;\n" ::"r"(dc_smem_addr(&full[i])) : "memory");
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory");
    }
    __syncthreads();
    auto fetch = [&](int c) {                        // one thread: the operands of chunk c into their stage, as they lie in the buffer
        const unsigned char* rec = rec0 + (size_t)c * rec_step;
        unsigned char* st = dc_raw + (c % DC_STAGES) * dc_stage_bytes<DP>();
        uint64_t* bar = &full[c % DC_STAGES];
        constexpr int SLICE = DC_C * DC_VS * 4;
        asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;\n" ::"r"(dc_smem_addr(bar)), "r"(FIXED + SLICE) : "memory");
        dc_bulk_copy(st, rec, FIXED, bar);
        dc_bulk_copy(st + FIXED, rec + lay.u_off() + (size_t)blockIdx.x * SLICE, SLICE, bar);
    };
    if (tid == 0)
        for (int c = 0; c < DC_STAGES - 1 && c < n_chunks; ++c) fetch(c);
    // this warp's 16 rows of S; two column tiles of 8
    const bool owns = warp < DP / 16;
    float s[2][4];
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int row = 16 * warp + g + 8 * (e >> 1), col = v0 + 8 * j + 2 * t + (e & 1);
            s[j][e] = (row < D && col < V) ? S[(size_t)row * V + col] : 0.f;
        }
    auto publish = [&]() {                           // S as two planes, for the products of the next chunk
        if (!owns) return;
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                uint32_t hi, lo;
                lt_split2(s[j][2 * half], s[j][2 * half + 1], hi, lo);
                const int at = (16 * warp + g + 8 * half) * DC_SS + 8 * j + 2 * t;
                *reinterpret_cast<uint32_t*>(s_hi + at) = hi;
                *reinterpret_cast<uint32_t*>(s_lo + at) = lo;
            }
    };
    publish();
    const int mi = lane >> 3, lr = lane & 7;
    const int rt = warp & 3, ct = warp >> 2;         // row tile of [W; Q] (0, 1: W), column tile
    for (int c = 0; c < n_chunks; ++c) {
        const bool arrived = dc_wait(&full[c % DC_STAGES], (uint32_t)(c / DC_STAGES) & 1u, error);
        if (!__syncthreads_and(arrived)) {           // given up: the copies that are still under way end before the block does
            if (tid == 0)
                for (int k = c; k < min(c + DC_STAGES - 1, n_chunks); ++k) dc_wait(&full[k % DC_STAGES], (uint32_t)(k / DC_STAGES) & 1u, error);
            return;
        }
        // chunk c's operands and the planes of S are there; the stage of c - 1 is free
        if (tid == 0 && c + DC_STAGES - 1 < n_chunks) fetch(c + DC_STAGES - 1);
        const unsigned char* st = dc_raw + (c % DC_STAGES) * dc_stage_bytes<DP>();
        const __nv_bfloat16* planes = reinterpret_cast<const __nv_bfloat16*>(st);
        const __nv_bfloat16* b_hi = planes + 6 * DC_C * RS;
        const float* sp = reinterpret_cast<const float*>(b_hi + 2 * DC_C * DC_BS);
        const float* su = sp + DP;
        // ---- [W; Q] S ----
        float acc[3][4];                             // high x high, low x high, high x low
#pragma unroll
        for (int k = 0; k < 3; ++k) acc[k][0] = acc[k][1] = acc[k][2] = acc[k][3] = 0.f;
        const __nv_bfloat16* a_hi = planes + (rt >> 1) * 2 * DC_C * RS + 16 * (rt & 1) * RS;
        const __nv_bfloat16* a_lo = a_hi + DC_C * RS;
#pragma unroll
        for (int k2 = 0; k2 < DP / 32; ++k2) {       // 32 rows of S at a time: one transposing load per plane
            uint32_t bh[4], bl[4];
            const int b_at = (32 * k2 + lr + 8 * mi) * DC_SS + 8 * ct;
            lt_ldsm_x4_trans(bh, s_hi + b_at);
            lt_ldsm_x4_trans(bl, s_lo + b_at);
#pragma unroll
            for (int kk = 0; kk < 2; ++kk) {
                uint32_t ah[4], al[4];
                const int a_at = (lr + 8 * (mi & 1)) * RS + 32 * k2 + 16 * kk + 8 * (mi >> 1);
                dc_ldsm_x4(ah, a_hi + a_at);
                dc_ldsm_x4(al, a_lo + a_at);
                lt_mma(acc[0], ah, bh[2 * kk], bh[2 * kk + 1]);
                lt_mma(acc[1], al, bh[2 * kk], bh[2 * kk + 1]);
                lt_mma(acc[2], ah, bl[2 * kk], bl[2 * kk + 1]);
            }
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[0][e] += acc[1][e] + acc[2][e];
        if (rt < 2) {                                // u = U0 - W S
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int r = 16 * rt + g + 8 * half, cl = 8 * ct + 2 * t;
                const float2 u0 = *reinterpret_cast<const float2*>(su + r * DC_VS + cl);
                uint32_t hi, lo;
                lt_split2(u0.x - acc[0][2 * half], u0.y - acc[0][2 * half + 1], hi, lo);
                *reinterpret_cast<uint32_t*>(u_hi + r * DC_SS + cl) = hi;
                *reinterpret_cast<uint32_t*>(u_lo + r * DC_SS + cl) = lo;
            }
        }
        __syncthreads();                             // u is there; nobody reads the planes of S any more
        uint32_t uh[DC_C / 16][4], ul[DC_C / 16][4];
#pragma unroll
        for (int ks = 0; ks < DC_C / 16; ++ks) {
            const int at = (16 * ks + lr + 8 * (mi & 1)) * DC_SS + 8 * (mi >> 1);
            lt_ldsm_x4_trans(uh[ks], u_hi + at);
            lt_ldsm_x4_trans(ul[ks], u_lo + at);
        }
        // ---- S <- P S + K^T u ----
        if (owns) {
            const float p0 = sp[16 * warp + g], p1 = sp[16 * warp + g + 8];
            float add[2][2][4];                      // [column tile][high x high | mixed]
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int k = 0; k < 2; ++k) add[j][k][0] = add[j][k][1] = add[j][k][2] = add[j][k][3] = 0.f;
            const __nv_bfloat16* kt = planes + 4 * DC_C * RS;
#pragma unroll
            for (int ks = 0; ks < DC_C / 16; ++ks) {
                uint32_t ah[4], al[4];
                const int at = (16 * ks + lr + 8 * (mi >> 1)) * RS + 16 * warp + 8 * (mi & 1);
                lt_ldsm_x4_trans(ah, kt + at);
                lt_ldsm_x4_trans(al, kt + DC_C * RS + at);
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    lt_mma(add[j][0], ah, uh[ks][2 * j], uh[ks][2 * j + 1]);
                    lt_mma(add[j][1], al, uh[ks][2 * j], uh[ks][2 * j + 1]);
                    lt_mma(add[j][1], ah, ul[ks][2 * j], ul[ks][2 * j + 1]);
                }
            }
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) s[j][e] = fmaf(s[j][e], e < 2 ? p0 : p1, add[j][0][e] + add[j][1][e]);
            if (c + 1 < n_chunks) publish();
        }
        // ---- o = Q S + B u ----
        if (rt >= 2) {
            acc[1][0] = acc[1][1] = acc[1][2] = acc[1][3] = 0.f;
#pragma unroll
            for (int ks = 0; ks < DC_C / 16; ++ks) {
                uint32_t ah[4], al[4];
                const int at = (16 * (rt - 2) + lr + 8 * (mi & 1)) * DC_BS + 16 * ks + 8 * (mi >> 1);
                dc_ldsm_x4(ah, b_hi + at);
                dc_ldsm_x4(al, b_hi + DC_C * DC_BS + at);
                const uint32_t h0 = ct ? uh[ks][2] : uh[ks][0], h1 = ct ? uh[ks][3] : uh[ks][1];
                lt_mma(acc[0], ah, h0, h1);
                lt_mma(acc[1], al, h0, h1);
                lt_mma(acc[1], ah, ct ? ul[ks][2] : ul[ks][0], ct ? ul[ks][3] : ul[ks][1]);
            }
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int tok = first + c * DC_C + 16 * (rt - 2) + g + 8 * half;
                if (tok >= last) continue;
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int col = v0 + 8 * ct + 2 * t + e;
                    if (col < V) out[((size_t)tok * H + h) * V + col] = acc[0][2 * half + e] + acc[1][2 * half + e];
                }
            }
        }
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int row = 16 * warp + g + 8 * (e >> 1), col = v0 + 8 * j + 2 * t + (e & 1);
            if (row < D && col < V) S[(size_t)row * V + col] = s[j][e];
        }
    if (dc_extra_wait) dc_wait(&full[0], (uint32_t)((n_chunks + DC_STAGES - 1) / DC_STAGES) & 1u, error);
}

NI_EXPORT int ni_delta_chunk_set_wait(long long ticks, int extra_wait) {
    if (ticks <= 0) ticks = 2000000000LL;
    cudaError_t e = cudaMemcpyToSymbol(dc_wait_limit, &ticks, sizeof(ticks));
    if (e == cudaSuccess) e = cudaMemcpyToSymbol(dc_extra_wait, &extra_wait, sizeof(extra_wait));
    return e == cudaSuccess ? NI_OK : (int)e;
}

// Bytes of the buffer that ni_delta_chunk_recurrence needs.
NI_EXPORT long long ni_delta_chunk_buffer_bytes(int n_tokens, int n_seqs, int H, int D, int V) {
    if (D <= 0 || D > 128 || V <= 0) return 0;
    const DcLayout lay{dc_pad_dim(D), (V + DC_VS - 1) / DC_VS * DC_VS};
    return (long long)(n_tokens / DC_C + n_seqs) * H * (long long)lay.bytes();
}
NI_EXPORT int ni_delta_chunk_max_dim() { return 128; }

template <int DP, int TAPS>
static int dc_launch(const DcInput& in, float* state, int n_seqs, int max_q_len, void* buf, float* out, int* error,
                     cudaStream_t stream) {
    const DcLayout lay{DP, (in.V + DC_VS - 1) / DC_VS * DC_VS};
    const size_t smem_p = (size_t)(3 * DC_C * DP + 2 * DC_C * DC_AS + DC_C * lay.VP) * sizeof(float), smem_s = dc_scan_smem<DP>();
    static size_t configured = 0;
    if (configured < smem_p) {
        cudaError_t e = cudaFuncSetAttribute(delta_chunk_prepare_kernel<DP, TAPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_p);
        if (e == cudaSuccess)
            e = cudaFuncSetAttribute(delta_chunk_scan_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_s);
        if (e != cudaSuccess) return (int)e;
        configured = smem_p;
    }
    dim3 grid_p((max_q_len + DC_C - 1) / DC_C, in.H, n_seqs), grid_s(lay.VP / DC_VS, in.H, n_seqs);
    delta_chunk_prepare_kernel<DP, TAPS><<<grid_p, DC_THREADS, smem_p, stream>>>(in, (unsigned char*)buf, lay);
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) return (int)e;
    delta_chunk_scan_kernel<DP><<<grid_s, DC_THREADS, smem_s, stream>>>((const unsigned char*)buf, lay, state, in.state_stride,
                                                                        in.cu_q, in.slots, in.H, in.D, in.V, out, error);
    NI_RETURN_LAUNCH_STATUS();
}

// The rule over a step's prompt portions, from the projection (see DcInput) to the read-outs, out FP32 [T, H V]: the state
// [H, D, V] at the start of a request's row moves on; the convolution history behind it is read (ni_delta_gated_norm, which
// must follow, writes the new one).  error: a device int, zero on entry; non-zero afterwards if a wait inside the kernel ran
// out.  max_q_len: the most tokens a request brings.  buf: 16-byte aligned,
// ni_delta_chunk_buffer_bytes long.
NI_EXPORT int ni_delta_chunk_recurrence(const void* proj, int ld, int b_off, const float* conv_w, const float* a_log,
                                        const float* dt_bias, const float* z, int ld_z, float* state, long long state_stride,
                                        const int* cu_q, const int* slots, int n_tokens, int n_seqs, int max_q_len, int G, int H,
                                        int D, int V, int taps, void* buf, long long buf_bytes, float* out, int* error,
                                        cudaStream_t stream) {
    if (n_tokens <= 0 || n_seqs <= 0) return NI_OK;
    if (G <= 0 || H <= 0 || D <= 0 || V <= 0 || taps <= 0 || H % G || ld_z < H * D || max_q_len <= 0 || buf == nullptr || error == nullptr ||
        (reinterpret_cast<size_t>(buf) & 15) || buf_bytes < ni_delta_chunk_buffer_bytes(n_tokens, n_seqs, H, D, V) || b_off < 0 ||
        ld < b_off + H || ld < 2 * G * D + H * V || state_stride < (long long)H * D * V + (long long)(taps - 1) * (2 * G * D + H * V))
        return NI_ERR_BAD_ARGUMENT;
    if (D > 128 || V > 512 || H > 65535 || n_seqs > 65535) return NI_ERR_UNSUPPORTED_SIZE;
    const DcInput in = {(const __nv_bfloat16*)proj, conv_w, a_log, dt_bias, z, state, state_stride, cu_q, slots,
                        ld, b_off, ld_z, G, H, D, V, taps};
    const bool four = taps == 4 && (reinterpret_cast<size_t>(conv_w) & 15) == 0;
#define GO(DP)                                                                                    \
    return four ? dc_launch<DP, 4>(in, state, n_seqs, max_q_len, buf, out, error, stream)         \
                : dc_launch<DP, 0>(in, state, n_seqs, max_q_len, buf, out, error, stream)
    if (D <= 32) GO(32);
    if (D <= 64) GO(64);
    GO(128);
#undef GO
}
