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
// Two launches:
//   delta_chunk_prepare   per (chunk, head), all at once: A, B (a group of 8 lanes per s walks i upwards with k_s times the
//                         decays in registers - what is left at the end is the last line's factor), then a thread per column
//                         of [W | U0] does the substitution
//   delta_chunk_scan      per (request, head, 16 value columns): the chunks one after the other; S stands in the
//                         accumulators of its four warps, and as two bfloat16 planes in shared memory for the products that
//                         read it; the next chunk's operands are copied while this one's are used
// A chunk begins at a portion's first token, so where a prompt is cut changes results by roundings only.
#include "linear_attention.cuh"

#define DC_C 32          // tokens per chunk
#define DC_THREADS 256   // of the preparation
#define DC_SCAN_THREADS 128
#define DC_VS 16         // value columns per block of the scan
#define DC_AS 36         // row stride of A in shared memory
#define DC_BS (DC_C + 8) // row stride of the planes of B

// One (chunk, head) of the buffer, in bytes: W, Q, K as two bfloat16 planes each [DC_C][DP], the two planes of B
// [DC_C][DC_C], U0 FP32 [DC_C][VP], P_n FP32 [DP].
struct DcLayout {
    int DP, VP;
    __host__ __device__ size_t plane() const { return (size_t)DC_C * DP * 2; }
    __host__ __device__ size_t b_off() const { return 6 * plane(); }
    __host__ __device__ size_t u_off() const { return b_off() + 2 * DC_C * DC_C * 2; }
    __host__ __device__ size_t p_off() const { return u_off() + (size_t)DC_C * VP * 4; }
    __host__ __device__ size_t bytes() const { return p_off() + (size_t)DP * 4; }
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

// qkv FP32 [T, C] (q | k | v of every head, q and k unit vectors per head, q scaled), gates [T, H, 2] (beta second), decay
// [T, ld_z] (H D).  grid (chunks of the longest portion, H, requests).  DP: the padded key size; a lane owns DP / 32 groups
// of four channels.
template <int DP>
__global__ void __launch_bounds__(DC_THREADS)
delta_chunk_prepare_kernel(const float* __restrict__ qkv, const float* __restrict__ gates, const float* __restrict__ decay,
                           int ld_z, const int* __restrict__ cu_q, int G, int H, int D, int V, unsigned char* __restrict__ buf,
                           DcLayout lay) {
    constexpr int M = DP / 32;
    extern __shared__ __align__(16) float dc_smem[];
    float* sq = dc_smem;                       // [DC_C][DP]
    float* sk = sq + DC_C * DP;
    float* sg = sk + DC_C * DP;
    float* sA = sg + DC_C * DP;                // [DC_C][DC_AS], times beta of the row
    float* sB = sA + DC_C * DC_AS;             // [DC_C][DC_AS]
    __shared__ float beta[DC_C];
    __shared__ int base_scratch;
    const int seq = blockIdx.z, h = blockIdx.y;
    const int first = cu_q[seq] + blockIdx.x * DC_C, last = cu_q[seq + 1];
    if (first >= last) return;
    const int n = min(DC_C, last - first);
    const int g = h / (H / G), C = 2 * G * D + H * V;
    unsigned char* rec = buf + ((size_t)(dc_chunk_base(cu_q, seq, &base_scratch) + blockIdx.x) * H + h) * lay.bytes();
    const int tid = threadIdx.x;
    for (int i = tid; i < DC_C * DP; i += DC_THREADS) {
        const int r = i / DP, d = i - r * DP;
        const bool ok = r < n && d < D;
        const float* row = qkv + (size_t)(first + r) * C;
        sq[i] = ok ? row[g * D + d] : 0.f;
        sk[i] = ok ? row[G * D + g * D + d] : 0.f;
        sg[i] = ok ? decay[(size_t)(first + r) * ld_z + h * D + d] : 1.f;
    }
    for (int i = tid; i < DC_C * DC_AS; i += DC_THREADS) sA[i] = sB[i] = 0.f;
    if (tid < DC_C) beta[tid] = tid < n ? gates[((size_t)(first + tid) * H + h) * 2 + 1] : 0.f;
    __syncthreads();
    {
        // warp w: the tokens s = w, 15 - w, 16 + w, 31 - w (early and late ones together); 8 lanes each
        const int warp = tid >> 5, lane = tid & 31, q4 = lane >> 3, l = lane & 7;
        const int s = q4 == 0 ? warp : (q4 == 1 ? 15 - warp : (q4 == 2 ? 16 + warp : 31 - warp));
        float kp[4 * M];
#pragma unroll
        for (int m = 0; m < M; ++m) {
            const float4 v = *reinterpret_cast<const float4*>(sk + s * DP + 4 * (l + 8 * m));
            kp[4 * m] = v.x; kp[4 * m + 1] = v.y; kp[4 * m + 2] = v.z; kp[4 * m + 3] = v.w;
        }
        for (int i = warp; i < DC_C; ++i) {            // (every s of the warp is at least `warp`)
            float a = 0.f, b = 0.f;
            if (i >= s) {
#pragma unroll
                for (int m = 0; m < M; ++m) {
                    const int c = 4 * (l + 8 * m);
                    if (i > s) {
                        const float4 gg = *reinterpret_cast<const float4*>(sg + i * DP + c);
                        kp[4 * m] *= gg.x; kp[4 * m + 1] *= gg.y; kp[4 * m + 2] *= gg.z; kp[4 * m + 3] *= gg.w;
                    }
                    const float4 kk = *reinterpret_cast<const float4*>(sk + i * DP + c);
                    const float4 qq = *reinterpret_cast<const float4*>(sq + i * DP + c);
                    a = fmaf(kk.x, kp[4 * m], a); a = fmaf(kk.y, kp[4 * m + 1], a);
                    a = fmaf(kk.z, kp[4 * m + 2], a); a = fmaf(kk.w, kp[4 * m + 3], a);
                    b = fmaf(qq.x, kp[4 * m], b); b = fmaf(qq.y, kp[4 * m + 1], b);
                    b = fmaf(qq.z, kp[4 * m + 2], b); b = fmaf(qq.w, kp[4 * m + 3], b);
                }
            }
#pragma unroll
            for (int off = 4; off > 0; off >>= 1) {
                a += __shfl_xor_sync(0xffffffffu, a, off);
                b += __shfl_xor_sync(0xffffffffu, b, off);
            }
            if (l == 0 && i >= s) {
                if (i > s) sA[i * DC_AS + s] = a * beta[i];
                sB[i * DC_AS + s] = b;
            }
        }
        __nv_bfloat16* k_hi = reinterpret_cast<__nv_bfloat16*>(rec + 4 * lay.plane()) + s * DP;
        __nv_bfloat16* k_lo = k_hi + DC_C * DP;
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
        for (int i = tid; i < DC_C * DC_C; i += DC_THREADS)
            dc_store_split(b_hi + i, b_hi + DC_C * DC_C + i, sB[(i / DC_C) * DC_AS + i % DC_C]);
    }
    __nv_bfloat16* w_hi = reinterpret_cast<__nv_bfloat16*>(rec);
    __nv_bfloat16* w_lo = w_hi + DC_C * DP;
    __nv_bfloat16* q_hi = w_lo + DC_C * DP;
    __nv_bfloat16* q_lo = q_hi + DC_C * DP;
    float* u0 = reinterpret_cast<float*>(rec + lay.u_off());
    for (int col = tid; col < DP + lay.VP; col += DC_THREADS) {
        const bool is_k = col < DP;
        const int vc = col - DP;
        const bool live = is_k || vc < V;
        const float* vrow = qkv + (size_t)first * C + 2 * G * D + h * V + vc;
        float x[DC_C], P = 1.f;
#pragma unroll
        for (int i = 0; i < DC_C; ++i) {
            float rhs;
            if (is_k) {
                P *= sg[i * DP + col];
                rhs = sk[i * DP + col] * P;
                dc_store_split(q_hi + i * DP + col, q_lo + i * DP + col, sq[i * DP + col] * P);
            } else {
                rhs = live && i < n ? vrow[(size_t)i * C] : 0.f;
            }
            float acc0 = beta[i] * rhs, acc1 = 0.f;
#pragma unroll
            for (int s = 0; s < i; s += 4) {
                const float4 a = *reinterpret_cast<const float4*>(sA + i * DC_AS + s);      // zero from column i on
                acc0 = fmaf(-a.x, x[s], acc0);
                if (s + 1 < i) acc1 = fmaf(-a.y, x[s + 1], acc1);
                if (s + 2 < i) acc0 = fmaf(-a.z, x[s + 2], acc0);
                if (s + 3 < i) acc1 = fmaf(-a.w, x[s + 3], acc1);
            }
            x[i] = acc0 + acc1;
            if (is_k) dc_store_split(w_hi + i * DP + col, w_lo + i * DP + col, x[i]);
            else u0[i * lay.VP + vc] = x[i];
        }
        if (is_k) reinterpret_cast<float*>(rec + lay.p_off())[col] = P;
    }
}

__device__ __forceinline__ void dc_ldsm_x4(uint32_t (&r)[4], const void* p) {
    const uint32_t addr = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}

template <int DP> __host__ __device__ constexpr int dc_stage_bytes() {
    return 6 * DC_C * (DP + 8) * 2 + 2 * DC_C * DC_BS * 2 + DC_C * DC_VS * 4 + DP * 4;
}
#define DC_SS (DC_VS + 8)          // row stride of the planes of S and of u
template <int DP> __host__ __device__ constexpr int dc_scan_smem() { return 2 * dc_stage_bytes<DP>() + 2 * DP * DC_SS * 2 + 2 * DC_C * DC_SS * 2; }

// grid (value slices, H, requests); 4 warps.
template <int DP>
__global__ void __launch_bounds__(DC_SCAN_THREADS)
delta_chunk_scan_kernel(const unsigned char* __restrict__ buf, DcLayout lay, float* __restrict__ state, long long state_stride,
                        const int* __restrict__ cu_q, const int* __restrict__ slots, int H, int D, int V,
                        float* __restrict__ out) {
    constexpr int RS = DP + 8;                       // row stride of the operand planes
    constexpr int MT = DP / 16 < 4 ? 1 : DP / 64;    // row tiles of S per warp
    extern __shared__ __align__(16) unsigned char dc_raw[];
    __shared__ int base_scratch;
    const int seq = blockIdx.z, h = blockIdx.y, v0 = blockIdx.x * DC_VS;
    const int first = cu_q[seq], last = cu_q[seq + 1];
    if (first >= last) return;
    const int n_chunks = (last - first + DC_C - 1) / DC_C;
    const unsigned char* rec0 = buf + ((size_t)dc_chunk_base(cu_q, seq, &base_scratch) * H + h) * lay.bytes();
    const size_t rec_step = (size_t)H * lay.bytes();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    __nv_bfloat16* s_hi = reinterpret_cast<__nv_bfloat16*>(dc_raw + 2 * dc_stage_bytes<DP>());     // [DP][DC_SS]
    __nv_bfloat16* s_lo = s_hi + DP * DC_SS;
    __nv_bfloat16* u_hi = s_lo + DP * DC_SS;                                                         // [DC_C][DC_SS]
    __nv_bfloat16* u_lo = u_hi + DC_C * DC_SS;
    float* S = state + (size_t)slots[seq] * state_stride + (size_t)h * D * V;

    auto fetch = [&](int c) {                        // the operands of chunk c into their stage
        const unsigned char* rec = rec0 + (size_t)c * rec_step;
        unsigned char* st = dc_raw + (c & 1) * dc_stage_bytes<DP>();
        constexpr int PIECES = DP / 8;
        for (int i = tid; i < 6 * DC_C * PIECES; i += DC_SCAN_THREADS) {
            const int r = i / PIECES, p = i - r * PIECES;                    // r: row of plane r / DC_C
            lt_cp_async16(st + ((size_t)r * RS + 8 * p) * 2, rec + ((size_t)r * DP + 8 * p) * 2);
        }
        unsigned char* sb = st + 6 * DC_C * RS * 2;
        for (int i = tid; i < 2 * DC_C * (DC_C / 8); i += DC_SCAN_THREADS) {
            const int r = i / (DC_C / 8), p = i % (DC_C / 8);
            lt_cp_async16(sb + (r * DC_BS + 8 * p) * 2, rec + lay.b_off() + (r * DC_C + 8 * p) * 2);
        }
        unsigned char* su = sb + 2 * DC_C * DC_BS * 2;
        for (int i = tid; i < DC_C * (DC_VS / 4); i += DC_SCAN_THREADS) {
            const int r = i / (DC_VS / 4), p = i % (DC_VS / 4);
            lt_cp_async16(su + (r * DC_VS + 4 * p) * 4, rec + lay.u_off() + ((size_t)r * lay.VP + v0 + 4 * p) * 4);
        }
        unsigned char* sp = su + DC_C * DC_VS * 4;
        for (int i = tid; i < DP / 4; i += DC_SCAN_THREADS) lt_cp_async16(sp + 16 * i, rec + lay.p_off() + 16 * i);
    };
    fetch(0);
    lt_cp_async_commit();
    // this warp's rows of S: tiles warp, warp + 4; two column tiles of 8
    float s[MT][2][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int row = 16 * (warp + 4 * m) + g + 8 * (e >> 1), col = v0 + 8 * j + 2 * t + (e & 1);
                s[m][j][e] = (row < D && col < V) ? S[(size_t)row * V + col] : 0.f;
            }
    auto publish = [&]() {                           // S as two planes, for the products of the next chunk
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            if (warp + 4 * m >= DP / 16) continue;
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    uint32_t hi, lo;
                    lt_split2(s[m][j][2 * half], s[m][j][2 * half + 1], hi, lo);
                    const int at = (16 * (warp + 4 * m) + g + 8 * half) * DC_SS + 8 * j + 2 * t;
                    *reinterpret_cast<uint32_t*>(s_hi + at) = hi;
                    *reinterpret_cast<uint32_t*>(s_lo + at) = lo;
                }
        }
    };
    publish();
    const int mi = lane >> 3, lr = lane & 7;
    for (int c = 0; c < n_chunks; ++c) {
        lt_cp_async_wait<0>();
        __syncthreads();                             // chunk c's operands and the planes of S are there; the other stage is free
        if (c + 1 < n_chunks) fetch(c + 1);
        lt_cp_async_commit();
        const unsigned char* st = dc_raw + (c & 1) * dc_stage_bytes<DP>();
        const __nv_bfloat16* planes = reinterpret_cast<const __nv_bfloat16*>(st);
        const __nv_bfloat16* b_hi = planes + 6 * DC_C * RS;
        const float* su = reinterpret_cast<const float*>(b_hi + 2 * DC_C * DC_BS);
        const float* sp = su + DC_C * DC_VS;
        // ---- [W; Q] S: warps 0 and 1 the 32 rows of W, 2 and 3 those of Q ----
        float acc[2][2][4];                          // [high x high | the two mixed terms][column tile]
#pragma unroll
        for (int k = 0; k < 2; ++k)
#pragma unroll
            for (int j = 0; j < 2; ++j) acc[k][j][0] = acc[k][j][1] = acc[k][j][2] = acc[k][j][3] = 0.f;
        const __nv_bfloat16* a_hi = planes + (warp >> 1) * 2 * DC_C * RS + 16 * (warp & 1) * RS;
        const __nv_bfloat16* a_lo = a_hi + DC_C * RS;
#pragma unroll
        for (int kk = 0; kk < DP / 16; ++kk) {
            uint32_t ah[4], al[4], bh[4], bl[4];
            const int a_at = (lr + 8 * (mi & 1)) * RS + 16 * kk + 8 * (mi >> 1);
            const int b_at = (16 * kk + lr + 8 * (mi & 1)) * DC_SS + 8 * (mi >> 1);
            dc_ldsm_x4(ah, a_hi + a_at);
            dc_ldsm_x4(al, a_lo + a_at);
            lt_ldsm_x4_trans(bh, s_hi + b_at);
            lt_ldsm_x4_trans(bl, s_lo + b_at);
            lt_mma(acc[0][0], ah, bh[0], bh[1]);
            lt_mma(acc[0][1], ah, bh[2], bh[3]);
            lt_mma(acc[1][0], al, bh[0], bh[1]);
            lt_mma(acc[1][1], al, bh[2], bh[3]);
            lt_mma(acc[1][0], ah, bl[0], bl[1]);
            lt_mma(acc[1][1], ah, bl[2], bl[3]);
        }
        if (warp < 2) {                              // u = U0 - W S
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int r = 16 * warp + g + 8 * half, cl = 8 * j + 2 * t;
                    const float2 u0 = *reinterpret_cast<const float2*>(su + r * DC_VS + cl);
                    uint32_t hi, lo;
                    lt_split2(u0.x - (acc[0][j][2 * half] + acc[1][j][2 * half]),
                              u0.y - (acc[0][j][2 * half + 1] + acc[1][j][2 * half + 1]), hi, lo);
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
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            const int tile = warp + 4 * m;
            if (tile >= DP / 16) continue;
            const float p0 = sp[16 * tile + g], p1 = sp[16 * tile + g + 8];
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                s[m][j][0] *= p0; s[m][j][1] *= p0;
                s[m][j][2] *= p1; s[m][j][3] *= p1;
            }
            const __nv_bfloat16* kt = planes + 4 * DC_C * RS;
#pragma unroll
            for (int ks = 0; ks < DC_C / 16; ++ks) {
                uint32_t ah[4], al[4];
                const int at = (16 * ks + lr + 8 * (mi >> 1)) * RS + 16 * tile + 8 * (mi & 1);
                lt_ldsm_x4_trans(ah, kt + at);
                lt_ldsm_x4_trans(al, kt + DC_C * RS + at);
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    lt_mma(s[m][j], ah, uh[ks][2 * j], uh[ks][2 * j + 1]);
                    lt_mma(s[m][j], al, uh[ks][2 * j], uh[ks][2 * j + 1]);
                    lt_mma(s[m][j], ah, ul[ks][2 * j], ul[ks][2 * j + 1]);
                }
            }
        }
        if (c + 1 < n_chunks) publish();
        // ---- o = Q S + B u ----
        if (warp >= 2) {
#pragma unroll
            for (int ks = 0; ks < DC_C / 16; ++ks) {
                uint32_t ah[4], al[4];
                const int at = (16 * (warp - 2) + lr + 8 * (mi & 1)) * DC_BS + 16 * ks + 8 * (mi >> 1);
                dc_ldsm_x4(ah, b_hi + at);
                dc_ldsm_x4(al, b_hi + DC_C * DC_BS + at);
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    lt_mma(acc[0][j], ah, uh[ks][2 * j], uh[ks][2 * j + 1]);
                    lt_mma(acc[1][j], al, uh[ks][2 * j], uh[ks][2 * j + 1]);
                    lt_mma(acc[1][j], ah, ul[ks][2 * j], ul[ks][2 * j + 1]);
                }
            }
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int tok = first + c * DC_C + 16 * (warp - 2) + g + 8 * half;
                if (tok >= last) continue;
#pragma unroll
                for (int j = 0; j < 2; ++j)
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        const int col = v0 + 8 * j + 2 * t + e;
                        if (col < V) out[((size_t)tok * H + h) * V + col] = acc[0][j][2 * half + e] + acc[1][j][2 * half + e];
                    }
            }
        }
    }
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int row = 16 * (warp + 4 * m) + g + 8 * (e >> 1), col = v0 + 8 * j + 2 * t + (e & 1);
                if (row < D && col < V) S[(size_t)row * V + col] = s[m][j][e];
            }
}

// Bytes of the buffer that ni_delta_chunk_recurrence needs.
NI_EXPORT long long ni_delta_chunk_buffer_bytes(int n_tokens, int n_seqs, int H, int D, int V) {
    if (D <= 0 || D > 128 || V <= 0) return 0;
    const DcLayout lay{dc_pad_dim(D), (V + DC_VS - 1) / DC_VS * DC_VS};
    return (long long)(n_tokens / DC_C + n_seqs) * H * (long long)lay.bytes();
}
NI_EXPORT int ni_delta_chunk_max_dim() { return 128; }

template <int DP>
static int dc_launch(const float* qkv, const float* gates, const float* decay, int ld_z, float* state, long long state_stride,
                     const int* cu_q, const int* slots, int n_seqs, int max_q_len, int G, int H, int D, int V, void* buf,
                     float* out, cudaStream_t stream) {
    const DcLayout lay{DP, (V + DC_VS - 1) / DC_VS * DC_VS};
    const size_t smem_p = (size_t)(3 * DC_C * DP + 2 * DC_C * DC_AS) * sizeof(float), smem_s = dc_scan_smem<DP>();
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(delta_chunk_prepare_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_p);
        if (e == cudaSuccess)
            e = cudaFuncSetAttribute(delta_chunk_scan_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_s);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    dim3 grid_p((max_q_len + DC_C - 1) / DC_C, H, n_seqs), grid_s(lay.VP / DC_VS, H, n_seqs);
    delta_chunk_prepare_kernel<DP><<<grid_p, DC_THREADS, smem_p, stream>>>(qkv, gates, decay, ld_z, cu_q, G, H, D, V,
                                                                           (unsigned char*)buf, lay);
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) return (int)e;
    delta_chunk_scan_kernel<DP><<<grid_s, DC_SCAN_THREADS, smem_s, stream>>>((const unsigned char*)buf, lay, state, state_stride,
                                                                             cu_q, slots, H, D, V, out);
    NI_RETURN_LAUNCH_STATUS();
}

// The recurrence over a step's tokens: qkv, gates and decay as ni_delta_prepare leaves them (decays per channel); the state
// [H, D, V] at the start of a request's row moves on; out FP32 [T, H V].  max_q_len: the most tokens a request brings.  buf:
// 16-byte aligned, ni_delta_chunk_buffer_bytes long.
NI_EXPORT int ni_delta_chunk_recurrence(const float* qkv, const float* gates, const float* decay, int ld_z, float* state,
                                        long long state_stride, const int* cu_q, const int* slots, int n_tokens, int n_seqs,
                                        int max_q_len, int G, int H, int D, int V, void* buf, long long buf_bytes, float* out,
                                        cudaStream_t stream) {
    if (n_tokens <= 0 || n_seqs <= 0) return NI_OK;
    if (G <= 0 || H <= 0 || D <= 0 || V <= 0 || H % G || ld_z < H * D || max_q_len <= 0 || buf == nullptr ||
        (reinterpret_cast<size_t>(buf) & 15) || buf_bytes < ni_delta_chunk_buffer_bytes(n_tokens, n_seqs, H, D, V) ||
        state_stride < (long long)H * D * V)
        return NI_ERR_BAD_ARGUMENT;
    if (D > 128 || H > 65535 || n_seqs > 65535) return NI_ERR_UNSUPPORTED_SIZE;
#define GO(DP) return dc_launch<DP>(qkv, gates, decay, ld_z, state, state_stride, cu_q, slots, n_seqs, max_q_len, G, H, D, V, buf, out, stream)
    if (D <= 32) GO(32);
    if (D <= 64) GO(64);
    GO(128);
#undef GO
}
