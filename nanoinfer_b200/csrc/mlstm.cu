// Matrix memories with exponential gates (the mLSTM cell of xLSTM): linear attention whose decay and input strength are
// numbers of every token, kept in a stabilised form, with a normaliser beside the matrix.
//
//   q, k [H, D], v [H, V] come in `proj`;  per head and token a log input gate i = cap tanh((z_i + b_i) / cap) and a
//   log forget gate f = logsigmoid(cap tanh((z_f + b_f) / cap)), z FP32 in `gates`
//   m_t = max(f_t + m_(t-1), i_t)                                    (running maximum, 0 at a sequence's start)
//   S_t = exp(f_t + m_(t-1) - m_t) S_(t-1) + exp(i_t - m_t) k_t v_t^T;   n_t likewise with k_t alone
//   o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + 1e-6),          q scaled by `q_scale`
//
// A request's state is one FP32 row: per head a record [S (D V) | n (D) | pad to 4], then m of every head.  Everything
// after the projections is FP32; sums of f over a chunk, from which small differences are taken, are formed in FP64.
//
// A request's tokens of a step run in chunks of LT_C tokens.  With F_t the sum of f up to token t of the chunk, a_j = i_j -
// F_j and M_t = max(m_0, a_1 .. a_t), the recurrence written out is
//
//   m_t = F_t + M_t
//   o_t ~ sum_(j <= t) exp(a_j - M_t) (q_t . k_j) v_j + exp(m_0 - M_t) S_0^T q_t          (and the same with 1 for v_j and
//                                                                                          n_0 for S_0: n_t . q_t)
//   S_n = sum_j exp(a_j - M_n) k_j v_j^T + exp(m_0 - M_n) S_0
//
// where no exponent is ever positive.  Chunks depend on one another only through (S, n, m), so a step is three launches:
// every chunk's own sum relative to its own A = max_j a_j, a scan over the chunks, every chunk's read-out.  A step of
// single tokens is one launch that reads and writes every state once and finishes with the norm per head and the gate.
// bfloat16 projections whose sizes are multiples of 16 run on tensor cores: what is kept in 32 bits and read by a product
// - the weighted scores, the weighted keys of a chunk's sum, the state before a chunk - is split into two bfloat16 halves.
#include "linear_attention.cuh"

__host__ __device__ __forceinline__ long long ml_record(int D, int V) { return ((long long)D * V + D + 3) / 4 * 4; }

__device__ __forceinline__ float ml_capped(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float ml_log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// What a chunk's kernels need of its gates, in shared memory.  a and M as sums of two FP32 numbers (their difference is
// then exact to FP32 although F runs into the hundreds).
struct MlGates {
    float ah[LT_C], al[LT_C], mh[LT_C], ml[LT_C];
    float before[LT_C];          // exp(m_0 - M_t)
    float floor_[LT_C];          // exp(-m_t)
    double F;                    // the chunk's sum of f
};
__device__ __forceinline__ void ml_split(double x, float& hi, float& lo) {
    hi = (float)x;
    lo = isinf(hi) ? 0.f : (float)(x - (double)hi);
}
// The weight of token j in token t's read-out.
__device__ __forceinline__ float ml_weight(const MlGates& g, int j, int t) { return expf((g.ah[j] - g.mh[t]) + (g.al[j] - g.ml[t])); }

// By one warp; a lane has two neighbouring tokens.  zi, zf: the gates' columns of the chunk's first token.  m0 = -infinity
// leaves the state before the chunk out (M_t is then the chunk's own maximum).
__device__ __forceinline__ void ml_chunk_gates(const float* __restrict__ zi, const float* __restrict__ zf, int ld, float bi, float bf,
                                               float cap, int n, float m0, MlGates& g) {
    const int lane = threadIdx.x & 31;
    double f[2], a[2];
    float in[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const int t = 2 * lane + e;
        in[e] = -INFINITY;
        f[e] = 0.0;
        if (t < n) {
            in[e] = ml_capped(zi[(size_t)t * ld] + bi, cap);
            f[e] = (double)ml_log_sigmoid(ml_capped(zf[(size_t)t * ld] + bf, cap));
        }
    }
    double sum = f[0] + f[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const double v = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += v;
    }
    const double F1 = sum, F0 = sum - f[1];
    a[0] = (double)in[0] - F0;
    a[1] = (double)in[1] - F1;
    double top = fmax(a[0], a[1]);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const double v = __shfl_up_sync(0xffffffffu, top, o);
        if (lane >= o) top = fmax(top, v);
    }
    double prev = __shfl_up_sync(0xffffffffu, top, 1);
    if (lane == 0) prev = -INFINITY;
    const double M[2] = {fmax((double)m0, fmax(prev, a[0])), fmax((double)m0, top)};
    const double F[2] = {F0, F1};
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const int t = 2 * lane + e;
        ml_split(a[e], g.ah[t], g.al[t]);
        ml_split(M[e], g.mh[t], g.ml[t]);
        g.before[t] = expf((float)((double)m0 - M[e]));
        g.floor_[t] = expf((float)(-(F[e] + M[e])));
    }
    if (lane == 31) g.F = F1;              // tokens beyond the chunk's end add nothing
}

// A chunk's place: request, first token, tokens, number of the chunk in the step.
struct MlChunk { int c0, n, index; };
__device__ __forceinline__ bool ml_chunk(const int* __restrict__ cu_q, int seq, int chunk, int* scratch, MlChunk& c) {
    const int t0 = cu_q[seq], t1 = cu_q[seq + 1];
    c.c0 = t0 + chunk * LT_C;
    if (c.c0 >= t1) return false;
    c.index = lt_chunk_base(cu_q, seq, scratch) + chunk;
    c.n = min(LT_C, t1 - c.c0);
    return true;
}

// Where the gates of a step are: z [T, ld] FP32, columns col_i + head and col_f + head; biases [H].
struct MlGateArgs { const float* z; int ld, col_i, col_f; const float *bias_i, *bias_f; float cap; };
__device__ __forceinline__ void ml_gates_of(const MlGateArgs& a, int head, const MlChunk& c, float m0, MlGates& g) {
    const float* row = a.z + (size_t)c.c0 * a.ld;
    ml_chunk_gates(row + a.col_i + head, row + a.col_f + head, a.ld, a.bias_i[head], a.bias_f[head], a.cap, c.n, m0, g);
}

// ---- every chunk's own sum ---------------------------------------------------------------------------------------------
// sums [chunks, H, record]: sum_j exp(a_j - A) k_j v_j^T | sum_j exp(a_j - A) k_j;  meta [chunks, H] = (A, F).  The block
// of a request's first chunk copies the request's running maximum to m_before (the scan reads it there and writes the new
// one into the state, so no block reads what another one writes).
struct MlMeta { float A; double F; };

// grid (chunks of the longest request x row tiles x column tiles, H, requests)
template <typename T>
__global__ void __launch_bounds__(LT_THREADS)
mlstm_chunk_kv_kernel(const T* __restrict__ proj, int ld, const MlGateArgs gate, const float* __restrict__ state,
                      long long state_stride, const int* __restrict__ cu_q, const int* __restrict__ slots, float* __restrict__ sums,
                      MlMeta* __restrict__ meta, float* __restrict__ m_before, int H, int D, int V, int d_tiles, int v_tiles) {
    __shared__ __align__(16) float Ks[LT_C][LT_KV_TILE];
    __shared__ __align__(16) float Vs[LT_C][LT_KV_TILE];
    __shared__ MlGates g;
    __shared__ float w_rev[LT_C];            // weight of token LT_C - 1 - i (the tile loader scales row r by entry last - r)
    __shared__ int base_s;
    const int tid = threadIdx.x, head = blockIdx.y, seq = blockIdx.z;
    const int chunk = blockIdx.x / (d_tiles * v_tiles), tile = blockIdx.x % (d_tiles * v_tiles);
    const int d0 = (tile / v_tiles) * LT_KV_TILE, vt = tile % v_tiles, v0 = vt * LT_KV_TILE;
    MlChunk c;
    if (!ml_chunk(cu_q, seq, chunk, &base_s, c)) return;
    if (tid < 32) ml_gates_of(gate, head, c, -INFINITY, g);
    __syncthreads();
    const float A = g.mh[c.n - 1];
    if (tid < LT_C) w_rev[LT_C - 1 - tid] = tid < c.n ? expf((g.ah[tid] - A) + g.al[tid]) : 0.f;
    if (tid == 0 && tile == 0) {
        MlMeta* mt = meta + (size_t)c.index * H + head;
        mt->A = A;
        mt->F = g.F;
        if (chunk == 0) m_before[(size_t)c.index * H + head] = state[(size_t)slots[seq] * state_stride + (size_t)H * ml_record(D, V) + head];
    }
    __syncthreads();
    const int n = c.n;
    const T* row0 = proj + (size_t)c.c0 * ld;
    lt_load_tile<T, false>(row0 + (size_t)(H + head) * D + d0, ld, n, n, min(LT_KV_TILE, D - d0), LT_KV_TILE, &Ks[0][0], LT_KV_TILE, nullptr, 0);
    lt_load_tile<T, false>(row0 + (size_t)2 * H * D + (size_t)head * V + v0, ld, n, n, min(LT_KV_TILE, V - v0), LT_KV_TILE, &Vs[0][0],
                           LT_KV_TILE, w_rev, LT_C - 1);
    __syncthreads();
    const int vg = (tid % 16) * 4, dg = (tid / 16) * 4;
    float acc[4][4];
#pragma unroll
    for (int a = 0; a < 4; ++a)
#pragma unroll
        for (int b = 0; b < 4; ++b) acc[a][b] = 0.f;
    for (int j = 0; j < n; ++j) {
        const float4 k4 = *reinterpret_cast<const float4*>(&Ks[j][dg]);
        const float4 v4 = *reinterpret_cast<const float4*>(&Vs[j][vg]);
        const float kk[4] = {k4.x, k4.y, k4.z, k4.w}, vv[4] = {v4.x, v4.y, v4.z, v4.w};
#pragma unroll
        for (int a = 0; a < 4; ++a)
#pragma unroll
            for (int b = 0; b < 4; ++b) acc[a][b] = fmaf(kk[a], vv[b], acc[a][b]);
    }
    float* out = sums + ((size_t)c.index * H + head) * ml_record(D, V);
#pragma unroll
    for (int a = 0; a < 4; ++a)
#pragma unroll
        for (int b = 0; b < 4; ++b)
            if (d0 + dg + a < D && v0 + vg + b < V) out[(size_t)(d0 + dg + a) * V + v0 + vg + b] = acc[a][b];
    if (vt == 0 && tid < LT_KV_TILE && d0 + tid < D) {
        float s = 0.f;
        for (int j = 0; j < n; ++j) s = fmaf(w_rev[LT_C - 1 - j], Ks[j][tid], s);
        out[(size_t)D * V + d0 + tid] = s;
    }
}

// bfloat16 projections, D and V multiples of 16: grid (chunks of the longest request, H, requests); a warp owns 16 rows of
// the sum at a time, 64 columns at a time.
__global__ void __launch_bounds__(LT_THREADS)
mlstm_chunk_kv_tc_kernel(const __nv_bfloat16* __restrict__ proj, int ld, const MlGateArgs gate, const float* __restrict__ state,
                         long long state_stride, const int* __restrict__ cu_q, const int* __restrict__ slots,
                         float* __restrict__ sums, MlMeta* __restrict__ meta, float* __restrict__ m_before, int H, int D, int V) {
    extern __shared__ __align__(16) unsigned char ml_raw[];
    __shared__ MlGates g;
    __shared__ float w[LT_C];
    __shared__ int base_s;
    const int KS = D + 8, VS = V + 8;
    __nv_bfloat16* Khi = reinterpret_cast<__nv_bfloat16*>(ml_raw);      // [LT_C][KS] weighted keys
    __nv_bfloat16* Klo = Khi + LT_C * KS;
    __nv_bfloat16* Vs = Klo + LT_C * KS;                                // [LT_C][VS]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int chunk = blockIdx.x, head = blockIdx.y, seq = blockIdx.z;
    MlChunk c;
    if (!ml_chunk(cu_q, seq, chunk, &base_s, c)) return;
    const int n = c.n;
    const __nv_bfloat16* row0 = proj + (size_t)c.c0 * ld;
    lt_copy_raw<LT_THREADS>(row0 + (size_t)(H + head) * D, ld, n, LT_C, D, D, Khi, KS);
    lt_cp_async_commit();
    lt_copy_raw<LT_THREADS>(row0 + (size_t)2 * H * D + (size_t)head * V, ld, n, LT_C, V, V, Vs, VS);
    lt_cp_async_commit();
    if (warp == 0) {
        ml_gates_of(gate, head, c, -INFINITY, g);
        __syncwarp();
        const float A = g.mh[n - 1];
        for (int t = lane; t < LT_C; t += 32) w[t] = t < n ? expf((g.ah[t] - A) + g.al[t]) : 0.f;
        if (lane == 0) {
            MlMeta* mt = meta + (size_t)c.index * H + head;
            mt->A = A;
            mt->F = g.F;
            if (chunk == 0) m_before[(size_t)c.index * H + head] = state[(size_t)slots[seq] * state_stride + (size_t)H * ml_record(D, V) + head];
        }
    }
    lt_cp_async_wait<1>();                                 // this thread's keys are here; the values are still under way
    __syncthreads();
    lt_for_pieces<LT_THREADS>(LT_C, D, [&](int r, int col) {             // weighted in place, the remainders beside them
        uint4 raw = *reinterpret_cast<const uint4*>(Khi + r * KS + col), lo;
        const __nv_bfloat16* e = reinterpret_cast<const __nv_bfloat16*>(&raw);
        const float sc = w[r];
        float v[8];
#pragma unroll
        for (int k = 0; k < 8; ++k) v[k] = __bfloat162float(e[k]) * sc;
        lt_split2(v[0], v[1], raw.x, lo.x);
        lt_split2(v[2], v[3], raw.y, lo.y);
        lt_split2(v[4], v[5], raw.z, lo.z);
        lt_split2(v[6], v[7], raw.w, lo.w);
        *reinterpret_cast<uint4*>(Khi + r * KS + col) = raw;
        *reinterpret_cast<uint4*>(Klo + r * KS + col) = lo;
    });
    lt_cp_async_wait<0>();
    __syncthreads();
    const int gq = lane >> 2, tq = lane & 3, blk = lane >> 3, rr = lane & 7;
    const int k_steps = (n + 15) / 16;
    float* out = sums + ((size_t)c.index * H + head) * ml_record(D, V);
    const uint32_t ones = 0x3f803f80u;                     // two bfloat16 ones: the normaliser is a product with a column of them
    for (int mt = warp; mt < D / 16; mt += LT_THREADS / 32) {
        const int d0 = mt * 16;
        for (int vb = 0; vb < V; vb += 64) {
            const int pairs = min(4, (V - vb) / 16);
            float acc[8][4];
#pragma unroll
            for (int a = 0; a < 8; ++a)
#pragma unroll
                for (int b = 0; b < 4; ++b) acc[a][b] = 0.f;
            float accn[4] = {0.f, 0.f, 0.f, 0.f};
            for (int kt = 0; kt < k_steps; ++kt) {
                const int j0 = kt * 16;
                uint32_t ahi[4], alo[4];
                const int a_off = (j0 + (blk >> 1) * 8 + rr) * KS + d0 + (blk & 1) * 8;
                lt_ldsm_x4_trans(ahi, Khi + a_off);
                lt_ldsm_x4_trans(alo, Klo + a_off);
                if (vb == 0) {
                    lt_mma(accn, ahi, ones, ones);
                    lt_mma(accn, alo, ones, ones);
                }
                const __nv_bfloat16* vp = Vs + (j0 + (blk & 1) * 8 + rr) * VS + vb + (blk >> 1) * 8;
#pragma unroll
                for (int np = 0; np < 4; ++np) {
                    if (np < pairs) {
                        uint32_t b[4];
                        lt_ldsm_x4_trans(b, vp + np * 16);
                        lt_mma(acc[2 * np], ahi, b[0], b[1]);
                        lt_mma(acc[2 * np + 1], ahi, b[2], b[3]);
                        lt_mma(acc[2 * np], alo, b[0], b[1]);
                        lt_mma(acc[2 * np + 1], alo, b[2], b[3]);
                    }
                }
            }
            if (vb == 0 && tq == 0) {
                out[(size_t)D * V + d0 + gq] = accn[0];
                out[(size_t)D * V + d0 + gq + 8] = accn[2];
            }
#pragma unroll
            for (int nt = 0; nt < 8; ++nt) {
                if (nt < 2 * pairs) {
                    const int col = vb + nt * 8 + 2 * tq;
                    *reinterpret_cast<float2*>(out + (size_t)(d0 + gq) * V + col) = make_float2(acc[nt][0], acc[nt][1]);
                    *reinterpret_cast<float2*>(out + (size_t)(d0 + gq + 8) * V + col) = make_float2(acc[nt][2], acc[nt][3]);
                }
            }
        }
    }
}

// ---- the scan over a request's chunks --------------------------------------------------------------------------------------
// grid (ceil((D V + D) / threads), H, requests).  before [chunks, H, record]: the state before every chunk - FP32, or with
// `split` S as two bfloat16 planes [2, D, V] in the same bytes (n stays FP32); m_before [chunks, H] its running maximum
// (the first chunk's is there already).
__global__ void mlstm_scan_kernel(float* __restrict__ state, long long state_stride, const int* __restrict__ cu_q,
                                  const int* __restrict__ slots, const float* __restrict__ sums, const MlMeta* __restrict__ meta,
                                  float* __restrict__ before, float* __restrict__ m_before, int split, int H, int D, int V) {
    __shared__ int base_s;
    const int head = blockIdx.y, seq = blockIdx.z;
    const int len = cu_q[seq + 1] - cu_q[seq];
    if (len <= 0) return;
    const int base = lt_chunk_base(cu_q, seq, &base_s);
    const int e = blockIdx.x * blockDim.x + threadIdx.x, DV = D * V;
    const size_t rec = ml_record(D, V), stride = (size_t)H * rec, first = ((size_t)base * H + head) * rec;
    float* slot = state + (size_t)slots[seq] * state_stride;
    float* S = slot + (size_t)head * rec + e;
    // What happens at a chunk's end is the same for the whole head: the block's first warp works it out for 32 chunks at a
    // time - the chain of maxima in every lane alike, the two factors of chunk i in lane i.
    __shared__ float keep_s[32], take_s[32];
    const bool mine = e < DV + D;
    float s = mine ? *S : 0.f, m = m_before[(size_t)base * H + head];
    const float* own_p = sums + first + e;
    float* o32 = before + first + e;
    __nv_bfloat16* o16 = reinterpret_cast<__nv_bfloat16*>(before + first) + e;
    const bool planes = split && e < DV;
    const int chunks = (len + LT_C - 1) / LT_C;
    for (int g0 = 0; g0 < chunks; g0 += 32) {
        const int there = min(32, chunks - g0);
        if (threadIdx.x < 32) {
            const int lane = threadIdx.x;
            const MlMeta mt = lane < there ? meta[(size_t)(base + g0 + lane) * H + head] : MlMeta{0.f, 0.0};
            float m_old = 0.f, M_own = 0.f;
            for (int i = 0; i < there; ++i) {
                const float M = fmaxf(m, __shfl_sync(0xffffffffu, mt.A, i));
                if (lane == i) { m_old = m; M_own = M; }
                m = (float)(__shfl_sync(0xffffffffu, mt.F, i) + (double)M);
            }
            keep_s[lane] = expf(m_old - M_own);
            take_s[lane] = expf(mt.A - M_own);
            if (blockIdx.x == 0 && lane < there && g0 + lane > 0) m_before[(size_t)(base + g0 + lane) * H + head] = m_old;
        }
        __syncthreads();
        for (int c = 0; c < there && mine; c += 8) {
            float own[8];                         // loaded together: the chain below waits for memory once per group
#pragma unroll
            for (int i = 0; i < 8; ++i) own[i] = c + i < there ? own_p[(size_t)(g0 + c + i) * stride] : 0.f;
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                if (c + i >= there) break;
                const size_t at = (size_t)(g0 + c + i) * stride;
                if (planes) {
                    const __nv_bfloat16 hi = __float2bfloat16_rn(s);
                    o16[at * 2] = hi;
                    o16[at * 2 + DV] = __float2bfloat16_rn(s - __bfloat162float(hi));
                } else {
                    o32[at] = s;
                }
                s = fmaf(keep_s[c + i], s, take_s[c + i] * own[i]);
            }
        }
        __syncthreads();
    }
    if (mine) *S = s;
    if (blockIdx.x == 0 && threadIdx.x == 0) slot[(size_t)H * rec + head] = m;
}

// ---- every chunk's read-out -------------------------------------------------------------------------------------------------
// out FP32 [T, H V].  FP32 FMA loops; grid (chunks of the longest request x column tiles of VT, H, requests)
template <typename T, int VT>
__global__ void __launch_bounds__(LT_THREADS)
mlstm_chunk_out_kernel(const T* __restrict__ proj, int ld, const MlGateArgs gate, const int* __restrict__ cu_q,
                       const float* __restrict__ before, const float* __restrict__ m_before, float q_scale, float* __restrict__ out,
                       int H, int D, int V, int v_tiles) {
    extern __shared__ __align__(16) float sm[];
    __shared__ MlGates g;
    __shared__ float den[LT_C];
    __shared__ int base_s;
    constexpr int TT = LT_C * VT / (LT_THREADS * 4);        // tokens per thread of the read-out (4 columns each)
    constexpr int AS = LT_C + 4;
    const int DP = (D + 3) & ~3, QS = DP + 4;
    float* Ss = sm;                          // [DP][VT]
    float* Qs = Ss + DP * VT;                // [LT_C][QS]
    float* Ks = Qs + LT_C * QS;              // [LT_C][QS]
    float* Vs = Ks + LT_C * QS;              // [LT_C][VT]
    float* As = Vs + LT_C * VT;              // [LT_C][AS]
    float* ns = As + LT_C * AS;              // [DP] the normaliser before the chunk
    const int tid = threadIdx.x, head = blockIdx.y, seq = blockIdx.z;
    const int chunk = blockIdx.x / v_tiles, v0 = (blockIdx.x % v_tiles) * VT;
    MlChunk c;
    if (!ml_chunk(cu_q, seq, chunk, &base_s, c)) return;
    const int n = c.n, n4 = (n + 3) & ~3, vt = min(VT, V - v0);
    if (tid < 32) ml_gates_of(gate, head, c, m_before[(size_t)c.index * H + head], g);
    const float* rec0 = before + ((size_t)c.index * H + head) * ml_record(D, V);
    const T* row0 = proj + (size_t)c.c0 * ld;
    lt_load_tile<float, false>(rec0 + v0, V, D, DP, vt, VT, Ss, VT, nullptr, 0);
    lt_load_tile<T, false>(row0 + (size_t)head * D, ld, n, n4, D, DP, Qs, QS, nullptr, 0);
    lt_load_tile<T, false>(row0 + (size_t)(H + head) * D, ld, n, n4, D, DP, Ks, QS, nullptr, 0);
    lt_load_tile<T, false>(row0 + (size_t)2 * H * D + (size_t)head * V + v0, ld, n, n4, vt, VT, Vs, VT, nullptr, 0);
    for (int d = tid; d < DP; d += LT_THREADS) ns[d] = d < D ? rec0[(size_t)D * V + d] : 0.f;
    for (int i = tid; i < LT_C * AS; i += LT_THREADS) As[i] = 0.f;
    __syncthreads();
    // ---- weighted scores, zero above the diagonal; a thread owns one 4 x 4 tile on or below it
    if (tid < (LT_C / 4) * (LT_C / 4 + 1) / 2) {
        int ti = 0, ji = tid;
        while (ji > ti) { ji -= ti + 1; ++ti; }
        if (ti * 4 < n4) {
            float acc[4][4];
#pragma unroll
            for (int a = 0; a < 4; ++a)
#pragma unroll
                for (int b = 0; b < 4; ++b) acc[a][b] = 0.f;
            const float* qp = Qs + ti * 4 * QS;
            const float* kp = Ks + ji * 4 * QS;
            for (int d = 0; d < DP; d += 4) {
                float4 qv[4], kv[4];
#pragma unroll
                for (int a = 0; a < 4; ++a) {
                    qv[a] = *reinterpret_cast<const float4*>(qp + a * QS + d);
                    kv[a] = *reinterpret_cast<const float4*>(kp + a * QS + d);
                }
#pragma unroll
                for (int a = 0; a < 4; ++a)
#pragma unroll
                    for (int b = 0; b < 4; ++b) {
                        acc[a][b] = fmaf(qv[a].x, kv[b].x, acc[a][b]);
                        acc[a][b] = fmaf(qv[a].y, kv[b].y, acc[a][b]);
                        acc[a][b] = fmaf(qv[a].z, kv[b].z, acc[a][b]);
                        acc[a][b] = fmaf(qv[a].w, kv[b].w, acc[a][b]);
                    }
            }
#pragma unroll
            for (int a = 0; a < 4; ++a)
#pragma unroll
                for (int b = 0; b < 4; ++b) {
                    const int t = ti * 4 + a, j = ji * 4 + b;
                    As[t * AS + j] = (j <= t && t < n) ? acc[a][b] * q_scale * ml_weight(g, j, t) : 0.f;
                }
        }
    }
    __syncthreads();
    // ---- denominators: four neighbouring threads per token
    {
        const int t = tid >> 2, part = tid & 3;
        float own = 0.f, old = 0.f;
        if (t < n) {
            for (int j = part; j <= t; j += 4) own += As[t * AS + j];
            for (int d = part; d < D; d += 4) old = fmaf(ns[d], Qs[t * QS + d], old);
        }
        float nq = t < n ? fmaf(g.before[t] * q_scale, old, own) : 0.f;
        nq += __shfl_xor_sync(0xffffffffu, nq, 1);
        nq += __shfl_xor_sync(0xffffffffu, nq, 2);
        if (part == 0 && t < n) den[t] = fmaxf(fabsf(nq), g.floor_[t]) + 1e-6f;
    }
    __syncthreads();
    // ---- read-out; a thread owns TT tokens x 4 value columns
    const int vg = (tid % (VT / 4)) * 4, tg = (tid / (VT / 4)) * TT;
    if (tg >= n4) return;
    float intra[TT][4], inter[TT][4];
#pragma unroll
    for (int a = 0; a < TT; ++a)
#pragma unroll
        for (int b = 0; b < 4; ++b) intra[a][b] = inter[a][b] = 0.f;
    const int j_end = min((tg + TT + 3) & ~3, n4);             // scores beyond the diagonal are zero
    for (int j = 0; j < j_end; j += 4) {
        float4 av[TT], wv[4];
#pragma unroll
        for (int a = 0; a < TT; ++a) av[a] = *reinterpret_cast<const float4*>(As + (tg + a) * AS + j);
#pragma unroll
        for (int jj = 0; jj < 4; ++jj) wv[jj] = *reinterpret_cast<const float4*>(Vs + (j + jj) * VT + vg);
#pragma unroll
        for (int a = 0; a < TT; ++a) {
            const float aa[4] = {av[a].x, av[a].y, av[a].z, av[a].w};
#pragma unroll
            for (int jj = 0; jj < 4; ++jj) {
                intra[a][0] = fmaf(aa[jj], wv[jj].x, intra[a][0]);
                intra[a][1] = fmaf(aa[jj], wv[jj].y, intra[a][1]);
                intra[a][2] = fmaf(aa[jj], wv[jj].z, intra[a][2]);
                intra[a][3] = fmaf(aa[jj], wv[jj].w, intra[a][3]);
            }
        }
    }
    for (int d = 0; d < DP; d += 4) {
        float4 qv[TT], sv[4];
#pragma unroll
        for (int a = 0; a < TT; ++a) qv[a] = tg + a < n4 ? *reinterpret_cast<const float4*>(Qs + (tg + a) * QS + d) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int dd = 0; dd < 4; ++dd) sv[dd] = *reinterpret_cast<const float4*>(Ss + (d + dd) * VT + vg);
#pragma unroll
        for (int a = 0; a < TT; ++a) {
            const float qq[4] = {qv[a].x, qv[a].y, qv[a].z, qv[a].w};
#pragma unroll
            for (int dd = 0; dd < 4; ++dd) {
                inter[a][0] = fmaf(qq[dd], sv[dd].x, inter[a][0]);
                inter[a][1] = fmaf(qq[dd], sv[dd].y, inter[a][1]);
                inter[a][2] = fmaf(qq[dd], sv[dd].z, inter[a][2]);
                inter[a][3] = fmaf(qq[dd], sv[dd].w, inter[a][3]);
            }
        }
    }
#pragma unroll
    for (int a = 0; a < TT; ++a) {
        const int t = tg + a;
        if (t >= n) continue;
        float* o = out + (size_t)(c.c0 + t) * H * V + (size_t)head * V + v0 + vg;
        const float old = g.before[t] * q_scale, inv = 1.0f / den[t];
#pragma unroll
        for (int b = 0; b < 4; ++b)
            if (vg + b < vt) o[b] = fmaf(old, inter[a][b], intra[a][b]) * inv;
    }
}

// The norm per head and the gate, for a read-out that has a head's whole values: y = o / rms(o) * weight * sigmoid(gate).
struct MlNormArgs { const float* weight; float eps; int gate_col; };      // gate_col: the gate's first column in proj

// bfloat16 projections on tensor cores: grid (chunks of the longest request x column tiles of VT, H, requests); VT / 64
// groups of four warps, a group owns 64 columns, a warp of it 16 tokens of the chunk (the groups form the same scores).
// The values are copied into the keys' place where they fit, while the warps multiply with the state before the chunk.
// y null: the read-outs go to out, FP32; else (one tile holds a head's values) they are normed and gated into y.
template <int VT>
__global__ void __launch_bounds__(VT * 2, VT == 128 ? 2 : 3)
mlstm_chunk_out_tc_kernel(const __nv_bfloat16* __restrict__ proj, int ld, const MlGateArgs gate, const int* __restrict__ cu_q,
                          const float* __restrict__ before, const float* __restrict__ m_before, float q_scale, float* __restrict__ out,
                          __nv_bfloat16* __restrict__ y, const MlNormArgs norm, int H, int D, int V, int v_tiles, int v_in_k) {
    extern __shared__ __align__(16) unsigned char ml_raw[];
    __shared__ MlGates g;
    __shared__ float ss[VT / 64][LT_C];
    __shared__ int base_s;
    constexpr int VS = VT + 8, THREADS = VT * 2;
    const int QS = D + 8;
    __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(ml_raw);       // [LT_C][QS]
    __nv_bfloat16* Ks = Qs + LT_C * QS;                                 // [LT_C][QS]
    __nv_bfloat16* Shi = Ks + LT_C * QS;                                // [D][VS] the state before the chunk
    __nv_bfloat16* Slo = Shi + D * VS;
    float* ns = reinterpret_cast<float*>(Slo + D * VS);                 // [D] its normaliser
    __nv_bfloat16* Vs = v_in_k ? Ks : reinterpret_cast<__nv_bfloat16*>(ns + D);      // [LT_C][VS]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int head = blockIdx.y, seq = blockIdx.z;
    const int chunk = blockIdx.x / v_tiles, v0 = (blockIdx.x % v_tiles) * VT;
    MlChunk c;
    if (!ml_chunk(cu_q, seq, chunk, &base_s, c)) return;
    const int n = c.n, vt = min(VT, V - v0);
    const float* rec0 = before + ((size_t)c.index * H + head) * ml_record(D, V);
    const __nv_bfloat16* S0 = reinterpret_cast<const __nv_bfloat16*>(rec0) + v0;
    const __nv_bfloat16* row0 = proj + (size_t)c.c0 * ld;
    lt_copy_raw<THREADS>(row0 + (size_t)head * D, ld, n, LT_C, D, D, Qs, QS);
    lt_copy_raw<THREADS>(row0 + (size_t)(H + head) * D, ld, n, LT_C, D, D, Ks, QS);
    lt_cp_async_commit();
    lt_copy_raw<THREADS>(S0, V, D, D, vt, VT, Shi, VS);                            // the two planes of the state before
    lt_copy_raw<THREADS>(S0 + (size_t)D * V, V, D, D, vt, VT, Slo, VS);
    lt_cp_async_commit();
    for (int d = tid; d < D; d += THREADS) ns[d] = rec0[(size_t)D * V + d];
    if (warp == 0) ml_gates_of(gate, head, c, m_before[(size_t)c.index * H + head], g);
    lt_cp_async_wait<1>();                                 // q and k are here; the state's planes are still under way
    __syncthreads();
    const int mw = warp & 3, vg = warp >> 2, vh = vg * 64;             // the warp's tokens and its columns of the tile
    const bool active = mw * 16 < n && vh < vt;           // the others only copy and wait with the block
    const int pairs = min(4, max(0, vt - vh) / 16);
    const int gq = lane >> 2, tq = lane & 3, blk = lane >> 3, rr = lane & 7;
    const int r0 = mw * 16, ta = r0 + gq, tb = ta + 8;    // this lane's two tokens
    float sc[8][4], acc[8][4];
#pragma unroll
    for (int a = 0; a < 8; ++a)
#pragma unroll
        for (int b = 0; b < 4; ++b) sc[a][b] = acc[a][b] = 0.f;
    float nq[2] = {0.f, 0.f};                             // n_t . q_t of the two tokens, this lane's part
    if (active) {
        float old[2] = {0.f, 0.f};
        for (int kk = 0; kk < D; kk += 16) {
            uint32_t a[4];
            const __nv_bfloat16* qp = Qs + ta * QS + kk + 2 * tq;
            a[0] = *reinterpret_cast<const uint32_t*>(qp);
            a[1] = *reinterpret_cast<const uint32_t*>(qp + 8 * QS);
            a[2] = *reinterpret_cast<const uint32_t*>(qp + 8);
            a[3] = *reinterpret_cast<const uint32_t*>(qp + 8 * QS + 8);
            const float2 n0 = *reinterpret_cast<const float2*>(ns + kk + 2 * tq), n1 = *reinterpret_cast<const float2*>(ns + kk + 2 * tq + 8);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float2 qf = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a[e]));
                const float2 nf = e < 2 ? n0 : n1;
                old[e & 1] = fmaf(qf.x, nf.x, fmaf(qf.y, nf.y, old[e & 1]));
            }
#pragma unroll
            for (int nt = 0; nt < 8; ++nt) {
                if (nt < 2 * mw + 2) {
                    const __nv_bfloat16* kp = Ks + (nt * 8 + gq) * QS + kk + 2 * tq;
                    lt_mma(sc[nt], a, *reinterpret_cast<const uint32_t*>(kp), *reinterpret_cast<const uint32_t*>(kp + 8));
                }
            }
        }
        const float mha = g.mh[ta], mla = g.ml[ta], mhb = g.mh[tb], mlb = g.ml[tb];
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) {
            if (nt < 2 * mw + 2) {
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const int j = nt * 8 + 2 * tq + i;
                    const float ah = g.ah[j], al = g.al[j];
                    sc[nt][i] = j <= ta ? sc[nt][i] * q_scale * __expf((ah - mha) + (al - mla)) : 0.f;
                    sc[nt][2 + i] = j <= tb ? sc[nt][2 + i] * q_scale * __expf((ah - mhb) + (al - mlb)) : 0.f;
                    nq[0] += sc[nt][i];
                    nq[1] += sc[nt][2 + i];
                }
            }
        }
        nq[0] = fmaf(g.before[ta] * q_scale, old[0], nq[0]);
        nq[1] = fmaf(g.before[tb] * q_scale, old[1], nq[1]);
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        nq[e] += __shfl_xor_sync(0xffffffffu, nq[e], 1);
        nq[e] += __shfl_xor_sync(0xffffffffu, nq[e], 2);
    }
    lt_cp_async_wait<0>();
    __syncthreads();                                      // the state's planes are here; nobody reads the keys any more
    lt_copy_raw<THREADS>(row0 + (size_t)2 * H * D + (size_t)head * V + v0, ld, n, LT_C, vt, VT, Vs, VS);
    lt_cp_async_commit();
    if (active) {
        for (int kk = 0; kk < D; kk += 16) {              // what the state before the chunk gives
            uint32_t a[4];
            const __nv_bfloat16* qp = Qs + ta * QS + kk + 2 * tq;
            a[0] = *reinterpret_cast<const uint32_t*>(qp);
            a[1] = *reinterpret_cast<const uint32_t*>(qp + 8 * QS);
            a[2] = *reinterpret_cast<const uint32_t*>(qp + 8);
            a[3] = *reinterpret_cast<const uint32_t*>(qp + 8 * QS + 8);
#pragma unroll
            for (int np = 0; np < 4; ++np) {
                if (np < pairs) {
                    const int off = (kk + (blk & 1) * 8 + rr) * VS + vh + np * 16 + (blk >> 1) * 8;
                    uint32_t b[4];
                    lt_ldsm_x4_trans(b, Shi + off);
                    lt_mma(acc[2 * np], a, b[0], b[1]);
                    lt_mma(acc[2 * np + 1], a, b[2], b[3]);
                    lt_ldsm_x4_trans(b, Slo + off);
                    lt_mma(acc[2 * np], a, b[0], b[1]);
                    lt_mma(acc[2 * np + 1], a, b[2], b[3]);
                }
            }
        }
        const float pa = g.before[ta] * q_scale, pb = g.before[tb] * q_scale;
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) {
            acc[nt][0] *= pa;
            acc[nt][1] *= pa;
            acc[nt][2] *= pb;
            acc[nt][3] *= pb;
        }
    }
    lt_cp_async_wait<0>();
    __syncthreads();
    if (active) {
#pragma unroll
        for (int kt = 0; kt < 4; ++kt) {                  // what the chunk's own tokens give
            if (kt <= mw) {
                uint32_t ahi[4], alo[4];
                lt_split2(sc[2 * kt][0], sc[2 * kt][1], ahi[0], alo[0]);
                lt_split2(sc[2 * kt][2], sc[2 * kt][3], ahi[1], alo[1]);
                lt_split2(sc[2 * kt + 1][0], sc[2 * kt + 1][1], ahi[2], alo[2]);
                lt_split2(sc[2 * kt + 1][2], sc[2 * kt + 1][3], ahi[3], alo[3]);
#pragma unroll
                for (int np = 0; np < 4; ++np) {
                    if (np < pairs) {
                        uint32_t b[4];
                        lt_ldsm_x4_trans(b, Vs + (kt * 16 + (blk & 1) * 8 + rr) * VS + vh + np * 16 + (blk >> 1) * 8);
                        lt_mma(acc[2 * np], ahi, b[0], b[1]);
                        lt_mma(acc[2 * np], alo, b[0], b[1]);
                        lt_mma(acc[2 * np + 1], ahi, b[2], b[3]);
                        lt_mma(acc[2 * np + 1], alo, b[2], b[3]);
                    }
                }
            }
        }
        const float ia = 1.0f / (fmaxf(fabsf(nq[0]), g.floor_[ta]) + 1e-6f), ib = 1.0f / (fmaxf(fabsf(nq[1]), g.floor_[tb]) + 1e-6f);
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) {
            acc[nt][0] *= ia;
            acc[nt][1] *= ia;
            acc[nt][2] *= ib;
            acc[nt][3] *= ib;
        }
    }
    if (y == nullptr) {
        if (!active) return;
        float* o = out + (size_t)c.c0 * H * V + (size_t)head * V + v0;
        const size_t os = (size_t)H * V;
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) {
            if (nt < 2 * pairs) {
                const int col = vh + nt * 8 + 2 * tq;
                if (ta < n) *reinterpret_cast<float2*>(o + (size_t)ta * os + col) = make_float2(acc[nt][0], acc[nt][1]);
                if (tb < n) *reinterpret_cast<float2*>(o + (size_t)tb * os + col) = make_float2(acc[nt][2], acc[nt][3]);
            }
        }
        return;
    }
    // ---- a head's whole values are in this block: norm and gate
    float sa = 0.f, sb = 0.f;
    if (active) {
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) {                  // columns beyond the tile's are zero
            sa = fmaf(acc[nt][0], acc[nt][0], fmaf(acc[nt][1], acc[nt][1], sa));
            sb = fmaf(acc[nt][2], acc[nt][2], fmaf(acc[nt][3], acc[nt][3], sb));
        }
    }
    sa += __shfl_xor_sync(0xffffffffu, sa, 1);
    sa += __shfl_xor_sync(0xffffffffu, sa, 2);
    sb += __shfl_xor_sync(0xffffffffu, sb, 1);
    sb += __shfl_xor_sync(0xffffffffu, sb, 2);
    if (tq == 0) {
        ss[vg][ta] = sa;
        ss[vg][tb] = sb;
    }
    __syncthreads();
    if (!active) return;
    sa = sb = 0.f;
#pragma unroll
    for (int k = 0; k < VT / 64; ++k) {
        sa += ss[k][ta];
        sb += ss[k][tb];
    }
    const float ra = 1.0f / sqrtf(sa / (float)V + norm.eps), rb = 1.0f / sqrtf(sb / (float)V + norm.eps);
    const __nv_bfloat16* gt = row0 + norm.gate_col + (size_t)head * V;
    __nv_bfloat16* yo = y + (size_t)c.c0 * H * V + (size_t)head * V;
    const float* wt = norm.weight + (size_t)head * V;
#pragma unroll
    for (int nt = 0; nt < 8; ++nt) {
        if (nt < 2 * pairs) {
            const int col = vh + nt * 8 + 2 * tq;
            const float2 wv = *reinterpret_cast<const float2*>(wt + col);
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int t = e ? tb : ta;
                if (t >= n) continue;
                const float2 z = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gt + (size_t)t * ld + col));
                const float r = e ? rb : ra;
                const float y0 = acc[nt][2 * e] * r * wv.x * __fdividef(1.0f, 1.0f + __expf(-z.x));
                const float y1 = acc[nt][2 * e + 1] * r * wv.y * __fdividef(1.0f, 1.0f + __expf(-z.y));
                *reinterpret_cast<__nv_bfloat162*>(yo + (size_t)t * H * V + col) = __floats2bfloat162_rn(y0, y1);
            }
        }
    }
}

// ---- a step of single tokens ---------------------------------------------------------------------------------------------
// grid (H, requests): a block owns one head of one request - state update, read-out, norm per head and gate.  proj FP32
// [T, ld] with columns q (H D) | k (H D) | v (H V) | gate (H V) | ...; a warp owns every 8th row of S, a lane 4
// neighbouring columns, 128 columns at a time.  y in the activations' type.
template <typename T>
__global__ void __launch_bounds__(LT_THREADS)
mlstm_token_kernel(const float* __restrict__ proj, int ld, const MlGateArgs gate, float* __restrict__ state, long long state_stride,
                   const int* __restrict__ cu_q, const int* __restrict__ slots, float q_scale, const MlNormArgs norm,
                   T* __restrict__ y, int H, int D, int V) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float scratch[32];
    float* qs = sm;                          // [D]
    float* ks = qs + D;                      // [D]
    float* part = ks + D;                    // [8 warps][128 columns]
    float* os = part + (LT_THREADS / 32) * 128;      // [V]
    constexpr int WARPS = LT_THREADS / 32, ROWS = 8;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int head = blockIdx.x, seq = blockIdx.y;
    const int t = cu_q[seq];
    if (cu_q[seq + 1] <= t) return;
    const float* row = proj + (size_t)t * ld;
    float* slot = state + (size_t)slots[seq] * state_stride;
    const size_t rec = ml_record(D, V);
    float* S = slot + (size_t)head * rec;
    float* N = S + (size_t)D * V;
    float* mp = slot + (size_t)H * rec + head;
    const float m_old = *mp;
    const float* z = gate.z + (size_t)t * gate.ld;
    const float i_log = ml_capped(z[gate.col_i + head] + gate.bias_i[head], gate.cap);
    const float f_log = ml_log_sigmoid(ml_capped(z[gate.col_f + head] + gate.bias_f[head], gate.cap));
    const float m_new = fmaxf(f_log + m_old, i_log);
    const float keep = expf(f_log + m_old - m_new), take = expf(i_log - m_new);
    float nq = 0.f;
    for (int d = tid; d < D; d += LT_THREADS) {
        const float q = row[(size_t)head * D + d] * q_scale, k = row[(size_t)(H + head) * D + d];
        qs[d] = q;
        ks[d] = take * k;
        const float nn = fmaf(keep, N[d], take * k);
        N[d] = nn;
        nq = fmaf(nn, q, nq);
    }
    nq = ni_block_sum(nq, scratch);          // (its barriers also order qs, ks and the reads of m)
    if (tid == 0) *mp = m_new;
    const float inv_den = 1.0f / (fmaxf(fabsf(nq), expf(-m_new)) + 1e-6f);
    float sq = 0.f;
    for (int v0 = 0; v0 < V; v0 += 128) {
        const int vc = v0 + lane * 4;
        float vv[4], acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int b = 0; b < 4; ++b) vv[b] = vc + b < V ? row[(size_t)2 * H * D + (size_t)head * V + vc + b] : 0.f;
        const bool wide = (V % 4 == 0) && ((reinterpret_cast<size_t>(S) & 15) == 0) && vc + 3 < V;
        if (wide) {
            for (int d = warp; d < D; d += ROWS * WARPS) {       // ROWS rows' loads are under way before the first store
                float4 s4[ROWS];
#pragma unroll
                for (int r = 0; r < ROWS; ++r)
                    if (d + r * WARPS < D) s4[r] = *reinterpret_cast<const float4*>(S + (size_t)(d + r * WARPS) * V + vc);
#pragma unroll
                for (int r = 0; r < ROWS; ++r) {
                    const int dr = d + r * WARPS;
                    if (dr >= D) break;
                    const float k = ks[dr], q = qs[dr];
                    s4[r].x = fmaf(keep, s4[r].x, k * vv[0]);
                    s4[r].y = fmaf(keep, s4[r].y, k * vv[1]);
                    s4[r].z = fmaf(keep, s4[r].z, k * vv[2]);
                    s4[r].w = fmaf(keep, s4[r].w, k * vv[3]);
                    *reinterpret_cast<float4*>(S + (size_t)dr * V + vc) = s4[r];
                    acc[0] = fmaf(s4[r].x, q, acc[0]);
                    acc[1] = fmaf(s4[r].y, q, acc[1]);
                    acc[2] = fmaf(s4[r].z, q, acc[2]);
                    acc[3] = fmaf(s4[r].w, q, acc[3]);
                }
            }
        } else {
            for (int d = warp; d < D; d += WARPS) {
                float* sp = S + (size_t)d * V + vc;
                const float k = ks[d], q = qs[d];
#pragma unroll
                for (int b = 0; b < 4; ++b)
                    if (vc + b < V) {
                        const float s1 = fmaf(keep, sp[b], k * vv[b]);
                        sp[b] = s1;
                        acc[b] = fmaf(s1, q, acc[b]);
                    }
            }
        }
        __syncthreads();                     // the partial sums of the tile before have been read
#pragma unroll
        for (int b = 0; b < 4; ++b) part[warp * 128 + lane * 4 + b] = acc[b];
        __syncthreads();
        if (tid < 128 && v0 + tid < V) {
            float o = 0.f;
#pragma unroll
            for (int w = 0; w < WARPS; ++w) o += part[w * 128 + tid];
            o *= inv_den;
            os[v0 + tid] = o;
            sq = fmaf(o, o, sq);
        }
    }
    sq = ni_block_sum(sq, scratch);
    const float inv = 1.0f / sqrtf(sq / (float)V + norm.eps);
    for (int v = tid; v < V; v += LT_THREADS) {
        const float gz = row[norm.gate_col + (size_t)head * V + v];
        y[(size_t)t * H * V + (size_t)head * V + v] =
            ni_from_float<T>(os[v] * inv * norm.weight[(size_t)head * V + v] * (1.0f / (1.0f + expf(-gz))));
    }
}

// ---- host side -----------------------------------------------------------------------------------------------------------
static long long ml_chunks(int n_tokens, int n_seqs) {          // the most chunks that requests of n_tokens tokens can have
    const long long whole = (long long)n_tokens / LT_C + n_seqs;
    return whole < n_tokens ? whole : n_tokens;
}
NI_EXPORT int ni_mlstm_max_chunks(int n_tokens, int n_seqs) { return (int)ml_chunks(n_tokens, n_seqs); }
// Floats of a request's state, and of the buffer of a step with prompt portions.
NI_EXPORT long long ni_mlstm_state_floats(int H, int D, int V) { return (long long)H * ml_record(D, V) + (H + 3) / 4 * 4; }
NI_EXPORT long long ni_mlstm_buffer_floats(int n_tokens, int n_seqs, int H, int D, int V) {
    return ml_chunks(n_tokens, n_seqs) * H * (2 * ml_record(D, V) + (long long)(sizeof(MlMeta) / sizeof(float)) + 1) + 8;
}

static bool ml_sizes_ok(int H, int D, int V, int ld, long long state_stride) {
    return H > 0 && D > 0 && V > 0 && ld >= 2 * H * D + 2 * H * V && state_stride >= ni_mlstm_state_floats(H, D, V) && state_stride % 4 == 0;
}

// One token per request: proj FP32 [n_seqs, ld] (q | k | v | gate | ...), gates FP32 with row length gate_ld (they may be
// columns of proj); y [n_seqs, H V] of y_dtype.
NI_EXPORT int ni_mlstm_token_step(const float* proj, int ld, const float* gates, int gate_ld, int col_i, int col_f,
                                  const float* bias_i, const float* bias_f, float cap, float* state, long long state_stride,
                                  const int* cu_q, const int* slots, int n_seqs, float q_scale, const float* weight, float eps,
                                  void* y, int y_dtype, int H, int D, int V, cudaStream_t stream) {
    if (n_seqs <= 0) return NI_OK;
    if (!ml_sizes_ok(H, D, V, ld, state_stride) || !(cap > 0.f)) return NI_ERR_BAD_ARGUMENT;
    if (n_seqs > 65535) return NI_ERR_UNSUPPORTED_SIZE;
    const MlGateArgs ga = {gates, gate_ld, col_i, col_f, bias_i, bias_f, cap};
    const MlNormArgs na = {weight, eps, 2 * H * D + H * V};
    const size_t smem = ((size_t)2 * D + (LT_THREADS / 32) * 128 + V) * sizeof(float);
    if (smem > 48 * 1024) return NI_ERR_UNSUPPORTED_SIZE;
    dim3 grid(H, n_seqs);
    if (y_dtype == NI_DTYPE_F32)
        mlstm_token_kernel<float><<<grid, LT_THREADS, smem, stream>>>(proj, ld, ga, state, state_stride, cu_q, slots, q_scale, na, (float*)y, H, D, V);
    else if (y_dtype == NI_DTYPE_BF16)
        mlstm_token_kernel<__nv_bfloat16><<<grid, LT_THREADS, smem, stream>>>(proj, ld, ga, state, state_stride, cu_q, slots, q_scale, na,
                                                                             (__nv_bfloat16*)y, H, D, V);
    else
        return NI_ERR_BAD_ARGUMENT;
    NI_RETURN_LAUNCH_STATUS();
}

static size_t ml_out_smem_bytes(int D, int VT) {
    const int DP = (D + 3) & ~3;
    return ((size_t)DP * VT + 2 * (size_t)LT_C * (DP + 4) + (size_t)LT_C * VT + (size_t)LT_C * (LT_C + 4) + DP) * sizeof(float);
}

// Any step: proj [T, ld] of `dtype` with columns q (H D) | k (H D) | v (H V) | gate (H V) | ...; gates FP32.  The read-outs
// go to out FP32 [T, H V] - or, where the kernel can, normed and gated to y (of `dtype`), and *finished is set to 1.
// buf: ni_mlstm_buffer_floats(...) floats, 16-byte aligned.
NI_EXPORT int ni_mlstm_chunk_step(const void* proj, int dtype, int ld, const float* gates, int gate_ld, int col_i, int col_f,
                                  const float* bias_i, const float* bias_f, float cap, float* state, long long state_stride,
                                  const int* cu_q, const int* slots, int n_tokens, int n_seqs, int max_q_len, float q_scale,
                                  const float* weight, float eps, float* buf, long long buf_floats, float* out, void* y,
                                  int* finished, int H, int D, int V, cudaStream_t stream) {
    *finished = 0;
    if (n_tokens <= 0 || n_seqs <= 0) return NI_OK;
    if (!ml_sizes_ok(H, D, V, ld, state_stride) || !(cap > 0.f) || max_q_len <= 0 || !buf ||
        buf_floats < ni_mlstm_buffer_floats(n_tokens, n_seqs, H, D, V))
        return NI_ERR_BAD_ARGUMENT;
    if (dtype != NI_DTYPE_F32 && dtype != NI_DTYPE_BF16) return NI_ERR_BAD_ARGUMENT;
    if (H > 65535 || n_seqs > 65535 || ((size_t)buf & 15)) return NI_ERR_UNSUPPORTED_SIZE;
    const long long rec = ml_record(D, V), chunks = ml_chunks(n_tokens, n_seqs);
    float* sums = buf;
    float* before = sums + (size_t)chunks * H * rec;
    MlMeta* meta = reinterpret_cast<MlMeta*>(before + (size_t)chunks * H * rec);
    float* m_before = reinterpret_cast<float*>(meta + (size_t)chunks * H);
    const MlGateArgs ga = {gates, gate_ld, col_i, col_f, bias_i, bias_f, cap};
    const MlNormArgs na = {weight, eps, 2 * H * D + H * V};
    const int per_seq = (max_q_len + LT_C - 1) / LT_C;
    dim3 grid_scan((D * V + D + LT_THREADS - 1) / LT_THREADS, H, n_seqs);
    if (dtype == NI_DTYPE_BF16 && D % 16 == 0 && V % 16 == 0 && ld % 8 == 0 && ((size_t)proj & 15) == 0 && ((size_t)out & 7) == 0 &&
        ((size_t)y & 3) == 0 && ((size_t)weight & 7) == 0) {
        const size_t smem_kv = ((size_t)2 * LT_C * (D + 8) + (size_t)LT_C * (V + 8)) * sizeof(__nv_bfloat16);
        auto out_bytes = [&](int vt) {
            return ((size_t)2 * LT_C * (D + 8) + (size_t)2 * D * (vt + 8) + (D >= vt ? 0 : (size_t)LT_C * (vt + 8))) * sizeof(__nv_bfloat16) +
                   (size_t)D * sizeof(float);
        };
        const int VT = V > 64 && out_bytes(128) <= 160 * 1024 ? 128 : 64;
        const int v_in_k = D >= VT, vt_tiles = (V + VT - 1) / VT;
        const size_t smem_out = out_bytes(VT);
        if (smem_kv <= 200 * 1024 && smem_out <= 200 * 1024) {
            const __nv_bfloat16* p = (const __nv_bfloat16*)proj;
            __nv_bfloat16* yo = vt_tiles == 1 ? (__nv_bfloat16*)y : nullptr;
            cudaError_t e = cudaFuncSetAttribute(mlstm_chunk_kv_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_kv);
            if (e != cudaSuccess) return (int)e;
            mlstm_chunk_kv_tc_kernel<<<dim3(per_seq, H, n_seqs), LT_THREADS, smem_kv, stream>>>(p, ld, ga, state, state_stride, cu_q, slots, sums,
                                                                                                meta, m_before, H, D, V);
            mlstm_scan_kernel<<<grid_scan, LT_THREADS, 0, stream>>>(state, state_stride, cu_q, slots, sums, meta, before, m_before, 1, H, D, V);
            const dim3 grid(per_seq * vt_tiles, H, n_seqs);
            if (VT == 128) {
                e = cudaFuncSetAttribute(mlstm_chunk_out_tc_kernel<128>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_out);
                if (e != cudaSuccess) return (int)e;
                mlstm_chunk_out_tc_kernel<128><<<grid, 256, smem_out, stream>>>(p, ld, ga, cu_q, before, m_before, q_scale, out, yo, na, H, D, V,
                                                                               vt_tiles, v_in_k);
            } else {
                e = cudaFuncSetAttribute(mlstm_chunk_out_tc_kernel<64>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_out);
                if (e != cudaSuccess) return (int)e;
                mlstm_chunk_out_tc_kernel<64><<<grid, 128, smem_out, stream>>>(p, ld, ga, cu_q, before, m_before, q_scale, out, yo, na, H, D, V,
                                                                              vt_tiles, v_in_k);
            }
            *finished = yo != nullptr;
            NI_RETURN_LAUNCH_STATUS();
        }
    }
    const int VT = D <= 128 ? 64 : 32;
    const size_t smem = ml_out_smem_bytes(D, VT);
    if (smem > 220 * 1024) return NI_ERR_UNSUPPORTED_SIZE;
    const int d_tiles = (D + LT_KV_TILE - 1) / LT_KV_TILE, kv_tiles = (V + LT_KV_TILE - 1) / LT_KV_TILE, v_tiles = (V + VT - 1) / VT;
    const dim3 grid_kv(per_seq * d_tiles * kv_tiles, H, n_seqs), grid_out(per_seq * v_tiles, H, n_seqs);
#define LAUNCH_OUT(T, VT)                                                                                                           \
    do {                                                                                                                            \
        cudaError_t e = cudaFuncSetAttribute(mlstm_chunk_out_kernel<T, VT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        if (e != cudaSuccess) return (int)e;                                                                                        \
        mlstm_chunk_out_kernel<T, VT><<<grid_out, LT_THREADS, smem, stream>>>((const T*)proj, ld, ga, cu_q, before, m_before, q_scale, \
                                                                             out, H, D, V, v_tiles);                                \
    } while (0)
#define LAUNCH(T)                                                                                                                   \
    do {                                                                                                                            \
        mlstm_chunk_kv_kernel<T><<<grid_kv, LT_THREADS, 0, stream>>>((const T*)proj, ld, ga, state, state_stride, cu_q, slots, sums, meta, \
                                                                     m_before, H, D, V, d_tiles, kv_tiles);                         \
        mlstm_scan_kernel<<<grid_scan, LT_THREADS, 0, stream>>>(state, state_stride, cu_q, slots, sums, meta, before, m_before, 0, H, D, V); \
        if (VT == 64) LAUNCH_OUT(T, 64); else LAUNCH_OUT(T, 32);                                                                    \
    } while (0)
    if (dtype == NI_DTYPE_F32) LAUNCH(float);
    else LAUNCH(__nv_bfloat16);
#undef LAUNCH
#undef LAUNCH_OUT
    NI_RETURN_LAUNCH_STATUS();
}
