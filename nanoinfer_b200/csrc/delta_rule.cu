// The gated delta rule: a recurrent token mixer with a matrix state per head.
//
// Per head (state S [D, V] in FP32, carried from token to token of a request):
//     S *= decay;   e = beta * (v - k S);   S += outer(k, e);   y = q S        (k, q: rows of D; v, e, y: rows of V)
// with q and k unit vectors per head (q also times D^-1/2) and beta = sigmoid(b).  The decay is one number per head,
// exp(-exp(A_log) softplus(a + dt_bias)), or one per head and key channel (then it multiplies the rows of S), whose
// logits come from elsewhere (a product with two thin matrices).  q, k and v first pass a short causal convolution over
// time per channel and silu; the last taps-1 inputs of every channel are part of a request's state.
//
// The step's tokens arrive as ONE fused projection `proj` ([T, ld], FP32 or bfloat16) whose first columns are
//     [ q: G D | k: G D | v: H V ],   with b (H) and, one decay per head, a (H) at offsets the caller names
// (G heads of q/k, H heads of v; head h reads q/k head h / (H / G)).  A request's state is a flat
// FP32 vector [ S: H D V | history: (taps-1) C ] with C = 2 G D + H V, found through slots[].
//
// Three launches, all FP32 inside:
//   delta_prepare      per token: convolution + silu, unit norms, beta, decay
//   (delta_history     per request: the new last taps-1 inputs; extra blocks of the gated norm's launch, which
//                      comes after delta_prepare has read the old ones)
//   delta_recurrence   per (request, head, a few value columns): its tokens one after the other
//   delta_gated_norm   per token and head: o / rms(o) * weight * silu or sigmoid(gate)
// Prompt portions and single tokens are the same case; a token's result depends only on its own
// request's state and tokens, in a fixed order of operations, however the step is cut.
//
// A step of single tokens with decays per channel has a fourth kernel, delta_token_step, that does all of it - the thin
// second products of decay and gate included - in one launch.
#include "common.cuh"

struct DeltaDims {
    int G, H, D, V, taps, ld;  // ld: row stride of proj
    int b_off, a_off;          // columns of b and a in proj (a_off < 0: decays per channel)
    __host__ __device__ int C() const { return 2 * G * D + H * V; }
    __host__ __device__ size_t hist_off() const { return (size_t)H * D * V; }
};

__device__ __forceinline__ float dr_silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float dr_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float dr_softplus(float z) { return z > 20.0f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float dr_decay(float a_log, float logit) { return expf(-expf(a_log) * dr_softplus(logit)); }

// Convolution of channel c at token t: taps inputs ending at this token.  Inputs before the
// portion's first token come from the request's history, zeros before the sequence's start.
template <typename T>
__device__ __forceinline__ float dr_conv(const T* __restrict__ proj, const float* __restrict__ conv_w,
                                         const float* __restrict__ hist, const DeltaDims& dm, int t, int in_portion,
                                         int c) {
    float acc = 0.f;
    const int C = dm.C();
    for (int j = 0; j < dm.taps; ++j) {
        const int back = dm.taps - 1 - j;
        float x;
        if (back <= in_portion) x = ni_to_float(proj[(size_t)(t - back) * dm.ld + c]);
        else x = hist[(size_t)(dm.taps - 1 - (back - in_portion)) * C + c];
        acc = fmaf(conv_w[(size_t)c * dm.taps + j], x, acc);
    }
    return dr_silu(acc);
}

// qkv [T, C]: q (unit, times D^-1/2), k (unit), v after convolution and silu; gates [T, H, 2]: decay, beta.
// One warp per unit of work of a token: a q or k head (unit norm over its D channels), 128 channels of v, or - decays
// per channel - 128 logits of z [T, ld_z], which become decays in place; the first warp of a token also computes beta and
// the decays per head.  grid = (tokens, units / warps per block).
#define DP_WARPS 4
#define DP_VCHUNK 128
template <typename T>
__global__ void __launch_bounds__(DP_WARPS * 32)
delta_prepare_kernel(const T* __restrict__ proj, const float* __restrict__ conv_w,
                     const float* __restrict__ a_log, const float* __restrict__ dt_bias,
                     const float* __restrict__ state, long long state_stride,
                     const int* __restrict__ seq_of_token, const int* __restrict__ cu_q,
                     const int* __restrict__ slots, DeltaDims dm, float* __restrict__ qkv,
                     float* __restrict__ gates, float* __restrict__ z, int ld_z) {
    const int t = blockIdx.x;
    const int lane = threadIdx.x & 31;
    int unit = blockIdx.y * DP_WARPS + (threadIdx.x >> 5);
    const int C = dm.C(), HV = dm.H * dm.V, HD = dm.H * dm.D;
    const int n_units = 2 * dm.G + (HV + DP_VCHUNK - 1) / DP_VCHUNK;
    if (unit >= n_units) {
        unit -= n_units;
        if (z == nullptr || unit * DP_VCHUNK >= HD) return;
        float* row = z + (size_t)t * ld_z;
        for (int c = unit * DP_VCHUNK + lane; c < (unit + 1) * DP_VCHUNK && c < HD; c += 32)
            row[c] = dr_decay(a_log[c / dm.D], row[c] + dt_bias[c]);
        return;
    }
    const int seq = seq_of_token[t];
    const int in_portion = t - cu_q[seq];
    const float* hist = state + (size_t)slots[seq] * state_stride + dm.hist_off();
    float* out = qkv + (size_t)t * C;
    if (unit < 2 * dm.G) {
        const int c0 = unit * dm.D;
        float ss = 0.f;
        for (int i = lane; i < dm.D; i += 32) {
            const float y = dr_conv(proj, conv_w, hist, dm, t, in_portion, c0 + i);
            out[c0 + i] = y;
            ss += y * y;
        }
        ss = ni_warp_sum(ss);
        float r = 1.0f / sqrtf(ss + 1e-6f);
        if (unit < dm.G) r *= 1.0f / sqrtf((float)dm.D);
        for (int i = lane; i < dm.D; i += 32) out[c0 + i] *= r;   // each lane rescales what it wrote itself
    } else {
        const int c0 = 2 * dm.G * dm.D + (unit - 2 * dm.G) * DP_VCHUNK;
        for (int c = c0 + lane; c < c0 + DP_VCHUNK && c < C; c += 32)
            out[c] = dr_conv(proj, conv_w, hist, dm, t, in_portion, c);
    }
    if (unit == 0) {
        const T* row = proj + (size_t)t * dm.ld;
        for (int h = lane; h < dm.H; h += 32) {
            gates[((size_t)t * dm.H + h) * 2] =
                dm.a_off >= 0 ? dr_decay(a_log[h], ni_to_float(row[dm.a_off + h]) + dt_bias[h]) : 1.0f;
            gates[((size_t)t * dm.H + h) * 2 + 1] = dr_sigmoid(ni_to_float(row[dm.b_off + h]));
        }
    }
}

// The request's new history: its last taps-1 inputs.  One thread per channel walks j upwards, so a
// portion shorter than the history shifts the old entries in place (it reads index j + q_len > j).
template <typename T>
__device__ __forceinline__ void delta_history(const T* __restrict__ proj, float* __restrict__ state,
                                              long long state_stride, const int* __restrict__ cu_q,
                                              const int* __restrict__ slots, const DeltaDims& dm, int seq, int c) {
    const int C = dm.C();
    if (c >= C) return;
    const int first = cu_q[seq], q_len = cu_q[seq + 1] - first;
    float* hist = state + (size_t)slots[seq] * state_stride + dm.hist_off();
    for (int j = 0; j < dm.taps - 1; ++j) {
        const int idx = q_len - (dm.taps - 1 - j);      // index into the portion; negative: before it
        hist[(size_t)j * C + c] = idx >= 0 ? ni_to_float(proj[(size_t)(first + idx) * dm.ld + c]) : hist[(size_t)(j + q_len) * C + c];
    }
}

// One warp per (request, head, a few value columns).  The rows of a column of S are cut into chunks of 8;
// a lane keeps CHUNKS of them in registers and RG lanes share a column, so k S and q S are sums inside a
// lane followed by log2(RG) shuffles.  The order of every sum is fixed by the chunk numbers alone (8 rows in
// four interleaved chains, then a binary tree over the chunk index from its lowest bit up), so the two
// layouts launched below - few lanes per column for single tokens, whose cost is reading and writing S in
// whole 32-byte sectors, and more lanes per column for long portions, whose cost is the chain of dependent
// operations per token - give the same bits.  (Key size 128, 16 heads, measured: one request of 2,048 tokens
// 695 us with 4 lanes per column, 613 us with 8, 647 us with 16; a batch of 8 single tokens 8.7 / 11.2 / 27.8 us.)  Lanes of one row group sit side by side and read neighbouring
// columns.  No block barrier.  What a token brings (k, q, the warp's values, decay, beta) travels through a
// ring of tokens in shared memory, filled by asynchronous copies that run ahead of the arithmetic.
#define DR_MAX_STAGES 8

__device__ __forceinline__ void dr_copy4(float* dst_smem, const float* src) {
    const unsigned d = (unsigned)__cvta_generic_to_shared(dst_smem);
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d), "l"(src) : "memory");
}
__device__ __forceinline__ void dr_copy8(float* dst_smem, const float* src) {
    const unsigned d = (unsigned)__cvta_generic_to_shared(dst_smem);
    asm volatile("cp.async.ca.shared.global [%0], [%1], 8;" ::"r"(d), "l"(src) : "memory");
}
__device__ __forceinline__ void dr_copy16(float* dst_smem, const float* src) {
    const unsigned d = (unsigned)__cvta_generic_to_shared(dst_smem);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
}

// CHANNEL: the decays are one per row of S, decay [T, ld_z] with head h's D numbers from column h D on; they travel with k
// and q.  Otherwise they are the first number of a head's pair in gates.
template <int CHUNKS, int RG, bool CHANNEL>
__global__ void __launch_bounds__(32)
delta_recurrence_kernel(const float* __restrict__ qkv, const float* __restrict__ gates,
                        const float* __restrict__ decay, int ld_z,
                        float* __restrict__ state, long long state_stride, const int* __restrict__ cu_q,
                        const int* __restrict__ slots, DeltaDims dm, float* __restrict__ out) {
    constexpr int ROWS = 8 * CHUNKS, COLS = 32 / RG, DP = ROWS * RG;   // rows per lane; columns per warp; D rounded up
    constexpr int STAGE = 2 * DP + 12 + (CHANNEL ? DP : 0);   // k | q | v of the warp's columns (up to 8) | decay, beta, -, - | decays per row
    constexpr int STAGES = CHANNEL ? (DP >= 1024 ? 3 : (DP >= 512 ? 4 : DR_MAX_STAGES)) : (DP >= 1024 ? 4 : DR_MAX_STAGES);
    __shared__ __align__(16) float ring[STAGES][STAGE];
    const int lane = threadIdx.x, rg = lane / COLS, cl = lane % COLS;
    const int h = blockIdx.y, seq = blockIdx.z;
    const int col = blockIdx.x * COLS + cl;
    const bool live = col < dm.V;
    const int D = dm.D, C = dm.C(), row0 = rg * ROWS;
    const int g = h / (dm.H / dm.G);
    const int first = cu_q[seq], last = cu_q[seq + 1];
    if (first >= last) return;
    const bool wide = (D % 4 == 0) && (C % 4 == 0) && (!CHANNEL || ld_z % 4 == 0);        // rows of k, q and the decays start on 16-byte boundaries
    const bool padded = D != DP;                           // same for the whole launch
    const bool ragged = blockIdx.x * COLS + COLS > dm.V;   // same for the whole warp: some of its columns do not exist
    if (padded || ragged) {                                // entries that no copy ever writes
        for (int st = 0; st < STAGES; ++st) {
            for (int i = lane; i < DP; i += 32)
                if (i >= D) {
                    ring[st][i] = ring[st][DP + i] = 0.f;
                    if (CHANNEL) ring[st][2 * DP + 12 + i] = 0.f;
                }
            if (lane < COLS && !live) ring[st][2 * DP + lane] = 0.f;
        }
    }
    // Each lane's sources of the next token to fetch, advanced by a row per token; its place in the ring likewise.
    const float* row = qkv + (size_t)first * C;
    const float* k_src = row + (dm.G + g) * D + (wide ? 4 * lane : lane);
    const float* q_src = row + g * D + (wide ? 4 * lane : lane);
    const float* v_src = row + 2 * dm.G * D + h * dm.V + col;
    const float* g_src = gates + ((size_t)first * dm.H + h) * 2;
    const float* d_src = CHANNEL ? decay + (size_t)first * ld_z + h * D + (wide ? 4 * lane : lane) : nullptr;
    int fetch_t = first, fetch_stage = 0;
    auto fetch = [&]() {                                   // the next token into its stage (nothing past the portion)
        if (fetch_t < last) {
            float* sg = ring[fetch_stage];
            if (wide) {
#pragma unroll
                for (int m = 0; m < (DP + 127) / 128; ++m)
                    if (4 * lane + 128 * m < D) {
                        dr_copy16(sg + 4 * lane + 128 * m, k_src + 128 * m);
                        dr_copy16(sg + DP + 4 * lane + 128 * m, q_src + 128 * m);
                        if (CHANNEL) dr_copy16(sg + 2 * DP + 12 + 4 * lane + 128 * m, d_src + 128 * m);
                    }
            } else {
#pragma unroll
                for (int m = 0; m < DP / 32; ++m)
                    if (lane + 32 * m < D) {
                        dr_copy4(sg + lane + 32 * m, k_src + 32 * m);
                        dr_copy4(sg + DP + lane + 32 * m, q_src + 32 * m);
                        if (CHANNEL) dr_copy4(sg + 2 * DP + 12 + lane + 32 * m, d_src + 32 * m);
                    }
            }
            if (lane < COLS && live) dr_copy4(sg + 2 * DP + lane, v_src);        // rg == 0 here
            if (lane == 31) dr_copy8(sg + 2 * DP + 8, g_src);                   // decay, beta
            k_src += C; q_src += C; v_src += C; g_src += 2 * dm.H;
            if (CHANNEL) d_src += ld_z;
        }
        ++fetch_t;
        fetch_stage = fetch_stage + 1 == STAGES ? 0 : fetch_stage + 1;
        asm volatile("cp.async.commit_group;" ::: "memory");     // one group per token, empty or not
    };
    for (int p = 0; p < STAGES - 1; ++p) fetch();
    float* S = state + (size_t)slots[seq] * state_stride + ((size_t)h * D + row0) * dm.V + col;   // this lane's first row
    float s[ROWS];
    if (!padded && !ragged) {
        const float* sp = S;
#pragma unroll
        for (int j = 0; j < ROWS; ++j, sp += dm.V) s[j] = *sp;
    } else {
#pragma unroll
        for (int j = 0; j < ROWS; ++j) s[j] = (live && row0 + j < D) ? S[(size_t)j * dm.V] : 0.f;
    }
    float* orow = out + (size_t)first * dm.H * dm.V + h * dm.V + col;
    int cur_stage = 0;
    float o_pending = 0.f;
    for (int t = first; t < last; ++t) {
        asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 2) : "memory");   // this lane's copies of token t
        __syncwarp();                                                            // ... and the other lanes'
        fetch();                               // token t + STAGES - 1, into the stage that token t-1 has left
        const float* sg = ring[cur_stage];
        cur_stage = cur_stage + 1 == STAGES ? 0 : cur_stage + 1;
        const float* kc = sg + row0;
        const float* qc = sg + DP + row0;
        const float gd = sg[2 * DP + 8], b = sg[2 * DP + 9];
        const float v = sg[2 * DP + cl];
        float part[CHUNKS];
#pragma unroll
        for (int c = 0; c < CHUNKS; ++c) {
            const float4 ka = *reinterpret_cast<const float4*>(kc + 8 * c);
            const float4 kb = *reinterpret_cast<const float4*>(kc + 8 * c + 4);
            float* sc = s + 8 * c;
            if (CHANNEL) {
                const float4 ga = *reinterpret_cast<const float4*>(sg + 2 * DP + 12 + row0 + 8 * c);
                const float4 gb = *reinterpret_cast<const float4*>(sg + 2 * DP + 12 + row0 + 8 * c + 4);
                sc[0] *= ga.x; sc[1] *= ga.y; sc[2] *= ga.z; sc[3] *= ga.w;
                sc[4] *= gb.x; sc[5] *= gb.y; sc[6] *= gb.z; sc[7] *= gb.w;
            } else {
#pragma unroll
                for (int j = 0; j < 8; ++j) sc[j] *= gd;
            }
            const float d0 = fmaf(sc[4], kb.x, sc[0] * ka.x), d1 = fmaf(sc[5], kb.y, sc[1] * ka.y);
            const float d2 = fmaf(sc[6], kb.z, sc[2] * ka.z), d3 = fmaf(sc[7], kb.w, sc[3] * ka.w);
            part[c] = (d0 + d1) + (d2 + d3);
        }
#pragma unroll
        for (int w = 1; w < CHUNKS; w <<= 1)
#pragma unroll
            for (int c = 0; c < CHUNKS; c += 2 * w) part[c] += part[c + w];
        float dot = part[0];
        // the lanes' partial sums of this token's k S and of the token before's q S travel together: two
        // independent shuffles per level instead of two trees one after the other
#pragma unroll
        for (int off = COLS; off < 32; off <<= 1) {
            dot += __shfl_xor_sync(0xffffffffu, dot, off);
            o_pending += __shfl_xor_sync(0xffffffffu, o_pending, off);
        }
        if (t > first && rg == 0 && live) orow[0] = o_pending;
        if (t > first) orow += dm.H * dm.V;
        const float u = b * (v - dot);
#pragma unroll
        for (int c = 0; c < CHUNKS; ++c) {
            const float4 ka = *reinterpret_cast<const float4*>(kc + 8 * c);
            const float4 kb = *reinterpret_cast<const float4*>(kc + 8 * c + 4);
            const float4 qa = *reinterpret_cast<const float4*>(qc + 8 * c);
            const float4 qb = *reinterpret_cast<const float4*>(qc + 8 * c + 4);
            float* sc = s + 8 * c;
            sc[0] = fmaf(ka.x, u, sc[0]); sc[1] = fmaf(ka.y, u, sc[1]); sc[2] = fmaf(ka.z, u, sc[2]); sc[3] = fmaf(ka.w, u, sc[3]);
            sc[4] = fmaf(kb.x, u, sc[4]); sc[5] = fmaf(kb.y, u, sc[5]); sc[6] = fmaf(kb.z, u, sc[6]); sc[7] = fmaf(kb.w, u, sc[7]);
            const float o0 = fmaf(sc[4], qb.x, sc[0] * qa.x), o1 = fmaf(sc[5], qb.y, sc[1] * qa.y);
            const float o2 = fmaf(sc[6], qb.z, sc[2] * qa.z), o3 = fmaf(sc[7], qb.w, sc[3] * qa.w);
            part[c] = (o0 + o1) + (o2 + o3);
        }
#pragma unroll
        for (int w = 1; w < CHUNKS; w <<= 1)
#pragma unroll
            for (int c = 0; c < CHUNKS; c += 2 * w) part[c] += part[c + w];
        o_pending = part[0];                   // summed over the lanes while the next token's k S is
        __syncwarp();                          // every lane has left this stage before a later fetch refills it
    }
#pragma unroll
    for (int off = COLS; off < 32; off <<= 1) o_pending += __shfl_xor_sync(0xffffffffu, o_pending, off);
    if (rg == 0 && live) orow[0] = o_pending;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    if (!padded && !ragged) {
        float* sp = S;
#pragma unroll
        for (int j = 0; j < ROWS; ++j, sp += dm.V) *sp = s[j];
    } else if (live) {
#pragma unroll
        for (int j = 0; j < ROWS; ++j)
            if (row0 + j < D) S[(size_t)j * dm.V] = s[j];
    }
}

// y[t, h, :] = o[t, h, :] / sqrt(mean(o[t, h, :]^2) + eps) * weight * act(gate[t, h, :]) * scale, act silu or sigmoid; one
// warp per (t, h); gate and y have row strides of their own.  The blocks behind those (from norm_blocks on) write the
// requests' new convolution history: by now the preparation, which read the old one, has ended, and one launch less stands
// between two steps' products.
template <typename T, typename TP>
__global__ void delta_gated_norm_kernel(const float* __restrict__ o, const float* __restrict__ gate, int ld_gate,
                                        int sigmoid_gate, const float* __restrict__ weight, float eps, float scale,
                                        DeltaDims dm, int n_tokens, T* __restrict__ y, int ld_y, int norm_blocks,
                                        int hist_blocks_per_seq, const TP* __restrict__ proj, float* __restrict__ state,
                                        long long state_stride, const int* __restrict__ cu_q,
                                        const int* __restrict__ slots, int wide) {
    if ((int)blockIdx.x >= norm_blocks) {
        const int hb = blockIdx.x - norm_blocks;
        delta_history(proj, state, state_stride, cu_q, slots, dm, hb / hist_blocks_per_seq,
                      (hb % hist_blocks_per_seq) * blockDim.x + threadIdx.x);
        return;
    }
    const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (item >= (long long)n_tokens * dm.H) return;
    const int lane = threadIdx.x & 31;
    const int t = (int)(item / dm.H), h = (int)(item - (long long)t * dm.H);
    const float* orow = o + ((size_t)t * dm.H + h) * dm.V;
    const float* grow = gate + (size_t)t * ld_gate + h * dm.V;
    T* yrow = y + (size_t)t * ld_y + (size_t)h * dm.V;
    float ss = 0.f;
    if (wide) {                            // V = 128, all rows on 16 bytes: four neighbours per lane, both rows asked for at once
        const float4 v = *reinterpret_cast<const float4*>(orow + 4 * lane), g = *reinterpret_cast<const float4*>(grow + 4 * lane);
        const float4 w = *reinterpret_cast<const float4*>(weight + 4 * lane);
        ss = ni_warp_sum(v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w);
        const float f = scale / sqrtf(ss / (float)dm.V + eps);
        const auto act = [&](float z) { return sigmoid_gate ? dr_sigmoid(z) : dr_silu(z); };
        __align__(16) T out[4] = {ni_from_float<T>(v.x * f * w.x * act(g.x)), ni_from_float<T>(v.y * f * w.y * act(g.y)),
                    ni_from_float<T>(v.z * f * w.z * act(g.z)), ni_from_float<T>(v.w * f * w.w * act(g.w))};
        if (sizeof(T) == 4) *reinterpret_cast<float4*>(yrow + 4 * lane) = *reinterpret_cast<float4*>(out);
        else *reinterpret_cast<uint2*>(yrow + 4 * lane) = *reinterpret_cast<uint2*>(out);
        return;
    }
    for (int i = lane; i < dm.V; i += 32) ss += orow[i] * orow[i];
    ss = ni_warp_sum(ss);
    const float inv = 1.0f / sqrtf(ss / (float)dm.V + eps);
    for (int i = lane; i < dm.V; i += 32) {
        const float g = sigmoid_gate ? dr_sigmoid(grow[i]) * scale : dr_silu(grow[i]) * scale;
        yrow[i] = ni_from_float<T>(orow[i] * inv * weight[i] * g);
    }
}

static int dr_check(const DeltaDims& dm) {
    if (dm.G <= 0 || dm.H <= 0 || dm.D <= 0 || dm.V <= 0 || dm.taps <= 0 || dm.H % dm.G) return NI_ERR_BAD_ARGUMENT;
    if (dm.ld < dm.C() || (dm.b_off >= 0 && dm.ld < dm.b_off + dm.H) || (dm.a_off >= 0 && dm.ld < dm.a_off + dm.H))
        return NI_ERR_BAD_ARGUMENT;
    if (dm.D > 1024) return NI_ERR_UNSUPPORTED_SIZE;      // a warp holds whole columns of a head's state: 32 lanes x 32 rows
    return NI_OK;
}

// Convolution, activations, unit norms, beta and decay of the step's tokens (the new history is written by
// ni_delta_gated_norm, which every step runs after this).  a_off < 0: the decays are one per head and key channel; their
// logits, z [T, ld_z] (H D columns), become decays in place, dt_bias has H D entries.
NI_EXPORT int ni_delta_prepare(const void* proj, int proj_dtype, const float* conv_w, const float* a_log, const float* dt_bias,
                               float* state, long long state_stride, const int* seq_of_token, const int* cu_q,
                               const int* slots, int n_tokens, int n_seqs, int G, int H, int D, int V, int taps, int ld,
                               int b_off, int a_off, float* z, int ld_z, float* qkv, float* gates, cudaStream_t stream) {
    if (n_tokens <= 0) return NI_OK;
    DeltaDims dm{G, H, D, V, taps, ld, b_off, a_off};
    if (int rc = dr_check(dm)) return rc;
    if (b_off < 0 || (a_off < 0) != (z != nullptr) || (z && ld_z < H * D)) return NI_ERR_BAD_ARGUMENT;
    const int n_units = 2 * G + (H * V + DP_VCHUNK - 1) / DP_VCHUNK + (z ? (H * D + DP_VCHUNK - 1) / DP_VCHUNK : 0);
    dim3 pgrid(n_tokens, (n_units + DP_WARPS - 1) / DP_WARPS);
    if (pgrid.y > 65535) return NI_ERR_UNSUPPORTED_SIZE;
    if (proj_dtype == NI_DTYPE_F32)
        delta_prepare_kernel<float><<<pgrid, DP_WARPS * 32, 0, stream>>>((const float*)proj, conv_w, a_log, dt_bias, state,
                                                                         state_stride, seq_of_token, cu_q, slots, dm, qkv,
                                                                         gates, z, ld_z);
    else if (proj_dtype == NI_DTYPE_BF16)
        delta_prepare_kernel<__nv_bfloat16><<<pgrid, DP_WARPS * 32, 0, stream>>>((const __nv_bfloat16*)proj, conv_w, a_log,
                                                                                 dt_bias, state, state_stride, seq_of_token,
                                                                                 cu_q, slots, dm, qkv, gates, z, ld_z);
    else
        return NI_ERR_BAD_ARGUMENT;
    NI_RETURN_LAUNCH_STATUS();
}

// decay / ld_z: decays per channel as ni_delta_prepare leaves them in z, or null (then gates holds one per head).
NI_EXPORT int ni_delta_recurrence(const float* qkv, const float* gates, const float* decay, int ld_z, float* state,
                                  long long state_stride, const int* cu_q, const int* slots, int n_tokens, int n_seqs,
                                  int G, int H, int D, int V, float* out, cudaStream_t stream) {
    if (n_seqs <= 0) return NI_OK;
    DeltaDims dm{G, H, D, V, 1, 2 * G * D + H * V, -1, -1};
    if (int rc = dr_check(dm)) return rc;
    if (decay && ld_z < H * D) return NI_ERR_BAD_ARGUMENT;
    if (H > 65535 || n_seqs > 65535) return NI_ERR_UNSUPPORTED_SIZE;
#define LAUNCH(CHUNKS, RG)                                                                                       \
    do {                                                                                                         \
        dim3 grid((V + 32 / (RG) - 1) / (32 / (RG)), H, n_seqs);                                                 \
        if (decay)                                                                                               \
            delta_recurrence_kernel<CHUNKS, RG, true><<<grid, 32, 0, stream>>>(qkv, gates, decay, ld_z, state,    \
                                                                               state_stride, cu_q, slots, dm, out); \
        else                                                                                                     \
            delta_recurrence_kernel<CHUNKS, RG, false><<<grid, 32, 0, stream>>>(qkv, gates, nullptr, 0, state,    \
                                                                                state_stride, cu_q, slots, dm, out); \
    } while (0)
    // Lanes per column (RG): single tokens take the fewest (whole sectors of S); long portions take the fewest that
    // still give every scheduler a warp or so (3 warps per SM and more: measured at key size 128, one request of
    // 2,048 tokens, 16 heads: 695 / 613 / 647 us with 4 / 8 / 16 lanes; 8 heads: 16 lanes ahead of 8; 8 requests
    // of 512 tokens: 483 / 488 / 734 us).  The bits are the same whichever is taken.
    const bool long_portions = n_tokens >= 8 * n_seqs;
    const int chunks_total = D <= 32 ? 4 : D <= 64 ? 8 : D <= 128 ? 16 : D <= 256 ? 32 : D <= 512 ? 64 : 128;
    int rg = chunks_total / 4 < 4 ? 4 : chunks_total / 4;             // 4 chunks per lane (1 where D <= 32)
    if (long_portions)
        while (rg < 32 && rg < chunks_total &&
               (long long)n_seqs * H * ((V + 32 / rg - 1) / (32 / rg)) < 3LL * ni_sm_count())
            rg *= 2;
    switch (chunks_total * 100 + rg) {
        case 404: LAUNCH(1, 4); break;
        case 804: LAUNCH(2, 4); break;
        case 808: LAUNCH(1, 8); break;
        case 1604: LAUNCH(4, 4); break;
        case 1608: LAUNCH(2, 8); break;
        case 1616: LAUNCH(1, 16); break;
        case 3208: LAUNCH(4, 8); break;
        case 3216: LAUNCH(2, 16); break;
        case 3232: LAUNCH(1, 32); break;
        case 6416: LAUNCH(4, 16); break;
        case 6432: LAUNCH(2, 32); break;
        case 12832: LAUNCH(4, 32); break;
        default: return NI_ERR_UNSUPPORTED_SIZE;
    }
#undef LAUNCH
    NI_RETURN_LAUNCH_STATUS();
}

// The gated norm of the step's read-outs, and the requests' new convolution history (taps > 1) from proj.  gate: FP32 rows
// ld_gate apart; sigmoid_gate 0: silu; scale: one more factor; y rows ld_y apart.
NI_EXPORT int ni_delta_gated_norm(const float* o, const float* gate, int ld_gate, int sigmoid_gate, const float* weight,
                                  float eps, float scale, int n_tokens, int n_seqs, int G, int H, int D, int V, int taps,
                                  void* y, int y_dtype, int ld_y, const void* proj, int proj_dtype, int ld, float* state,
                                  long long state_stride, const int* cu_q, const int* slots, cudaStream_t stream) {
    if (n_tokens <= 0) return NI_OK;
    DeltaDims dm{G, H, D, V, taps, ld, -1, -1};
    if (int rc = dr_check(dm)) return rc;
    if (ld_gate < H * V || ld_y < H * V) return NI_ERR_BAD_ARGUMENT;
    const int warps = 4;
    const long long norm_blocks = ((long long)n_tokens * H + warps - 1) / warps;
    const int per_seq = taps > 1 ? (dm.C() + warps * 32 - 1) / (warps * 32) : 0;
    const long long blocks = norm_blocks + (long long)per_seq * n_seqs;
    if (blocks > 2147483647LL) return NI_ERR_UNSUPPORTED_SIZE;
    const auto aligned = [](const void* q) { return (reinterpret_cast<size_t>(q) & 15) == 0; };
    const int wide = V == 128 && y_dtype == NI_DTYPE_BF16 && ld_gate % 4 == 0 && ld_y % 8 == 0 && aligned(o) && aligned(gate) &&
                     aligned(weight) && aligned(y);
#define GO(T, TP)                                                                                                        \
    delta_gated_norm_kernel<T, TP><<<(int)blocks, warps * 32, 0, stream>>>(                                              \
        o, gate, ld_gate, sigmoid_gate, weight, eps, scale, dm, n_tokens, (T*)y, ld_y, (int)norm_blocks, per_seq,        \
        (const TP*)proj, state, state_stride, cu_q, slots, wide)
    if (y_dtype == NI_DTYPE_F32 && proj_dtype == NI_DTYPE_F32) GO(float, float);
    else if (y_dtype == NI_DTYPE_BF16 && proj_dtype == NI_DTYPE_F32) GO(__nv_bfloat16, float);
    else if (y_dtype == NI_DTYPE_BF16 && proj_dtype == NI_DTYPE_BF16) GO(__nv_bfloat16, __nv_bfloat16);
    else return NI_ERR_BAD_ARGUMENT;
#undef GO
    NI_RETURN_LAUNCH_STATUS();
}
// ---- a step of single tokens with decays per channel: everything between the projections in one launch -------------------
//
// One block of 16 warps per (head, request).  A warp owns every 16th row of S, a lane every 32nd column; S is read into
// registers first, before anything else is needed.  Meanwhile: the convolution of the head's q, k and v channels (a thread
// per channel), the thin second products of its D decay logits and V gate logits (a group of lanes per row of the weights, 16
// bytes each; the thin first products stand in shared memory), unit norms.  Then k S, the error,
// the update, q S and the gated norm; S is written back once.
// The convolution history of the value channels is moved on by their own block.  A query/key channel belongs to the H / G
// heads that share it: the last of their blocks to have read the old inputs (an atomic ticket per request and q/k head, left
// zero) moves them on.  No block waits for another.
#define DT_WARPS 16
struct DeltaTokenParams {
    const float* proj;                 // [T, ld] FP32: q | k | v | ... b at b_off, the thin first products at thin_off
    const __nv_bfloat16* w_decay;      // [H D, ra]
    const __nv_bfloat16* w_gate;       // [H V, rg]
    const float *conv_w, *a_log, *dt_bias, *norm_w;
    float* state;
    long long state_stride;
    const int *cu_q, *slots;
    int* tickets;                      // [requests, G], zero
    __nv_bfloat16* y;
    int ld_y, thin_off, ra, rg;
    float eps, scale;
};

// DR: rows of S per warp (D <= 16 DR); VC: columns per lane (V <= 32 VC).  EXACT: D and V are those bounds, taps 4.
// Everything that does not depend on this block's own results - S, weights, constants, the history - is asked for before the
// first barrier, so that the chain of dependent memory round trips is short.
template <int DR, int VC, bool EXACT>
__global__ void __launch_bounds__(DT_WARPS * 32, 1)
delta_token_kernel(const DeltaTokenParams p, const DeltaDims dm) {
    constexpr int DP = DT_WARPS * DR, VP = 32 * VC, U = 8;
    __shared__ float sq[DP], sk[DP], sg[DP], sv[VP], sgate[VP], su[VP], red[DT_WARPS][VP], scratch[32];
    __shared__ float unit[2];          // what q and k are multiplied by
    __shared__ int s_last;
    extern __shared__ __align__(16) float thin[];       // [ra + rg]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int h = blockIdx.x, seq = blockIdx.y;
    const int D = EXACT ? DP : dm.D, V = EXACT ? VP : dm.V, taps = EXACT ? 4 : dm.taps;
    const int G = dm.G, C = dm.C(), per = dm.H / G, g = h / per;
    const int t = p.cu_q[seq];
    float* st = p.state + (size_t)p.slots[seq] * p.state_stride;
    float* S = st + (size_t)h * D * V;
    float* hist = st + (size_t)dm.H * D * V;
    float s[DR][VC];
#pragma unroll
    for (int i = 0; i < DR; ++i)
#pragma unroll
        for (int j = 0; j < VC; ++j) {
            const int row = warp + DT_WARPS * i, col = lane + 32 * j;
            s[i][j] = (EXACT || (row < D && col < V)) ? S[(size_t)row * V + col] : 0.f;
        }
    // the thin second products: the first half of the warps the D rows of the decay's matrix, the others the V rows of the
    // gate's; L lanes share a row, a lane's first 16 bytes of up to U rows are asked for here
    const bool gates = warp >= DT_WARPS / 2;
    const int n_thin = gates ? p.rg : p.ra, rows = gates ? V : D, w8 = warp & (DT_WARPS / 2 - 1);
    const int L = n_thin > 64 ? 16 : (n_thin > 32 ? 8 : 4), l = lane & (L - 1), sub = lane / L, per_warp = 32 / L;
    const __nv_bfloat16* w_thin = gates ? p.w_gate + (size_t)h * V * p.rg : p.w_decay + (size_t)h * D * p.ra;
    uint4 raw[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
        const int row = (u * (DT_WARPS / 2) + w8) * per_warp + sub;
        raw[u] = row < rows && 8 * l < n_thin ? *reinterpret_cast<const uint4*>(w_thin + (size_t)row * n_thin + 8 * l)
                                              : make_uint4(0u, 0u, 0u, 0u);
    }
    const float* row = p.proj + (size_t)t * dm.ld;
    const float a_log = p.a_log[h], beta = dr_sigmoid(row[dm.b_off + h]);
    const float dt = tid < D ? p.dt_bias[h * D + tid] : 0.f, norm_w = tid < V ? p.norm_w[tid] : 0.f;
    for (int i = tid; i < p.ra + p.rg; i += blockDim.x) thin[i] = row[p.thin_off + i];
    // the convolution: a thread per channel (2 D + V <= 384 < blockDim.x)
    int c = -1;
    float x = 0.f, h0 = 0.f, h1 = 0.f, h2 = 0.f;
    if (tid < 2 * D + V) {
        c = tid < D ? g * D + tid : (tid < 2 * D ? G * D + g * D + tid - D : 2 * G * D + h * V + tid - 2 * D);
        x = row[c];
        float acc = 0.f;
        if (EXACT) {                       // (taps 4: the weights in one load)
            const float4 w = *reinterpret_cast<const float4*>(p.conv_w + (size_t)c * 4);
            h0 = hist[c]; h1 = hist[(size_t)C + c]; h2 = hist[2 * (size_t)C + c];
            acc = fmaf(w.w, x, fmaf(w.z, h2, fmaf(w.y, h1, w.x * h0)));
        } else {
            for (int j = 0; j + 1 < taps; ++j) acc = fmaf(p.conv_w[(size_t)c * taps + j], hist[(size_t)j * C + c], acc);
            acc = fmaf(p.conv_w[(size_t)c * taps + taps - 1], x, acc);
        }
        const float y = dr_silu(acc);
        if (tid < D) sq[tid] = y;
        else if (tid < 2 * D) sk[tid - D] = y;
        else sv[tid - 2 * D] = y;
    }
    __syncthreads();
    if (tid == 0 && taps > 1) {
        int last = 1;
        if (per > 1) {
            __threadfence();
            int* ticket = p.tickets + (size_t)seq * G + g;
            last = atomicAdd(ticket, 1) == per - 1;
            if (last) *ticket = 0;
        }
        s_last = last;
    }
    {
        const float* xs = thin + (gates ? p.ra : 0);
        float a[U];
#pragma unroll
        for (int u = 0; u < U; ++u) a[u] = 0.f;
        for (int k = 8 * l; k < n_thin; k += 8 * L) {
            if (k != 8 * l) {
#pragma unroll
                for (int u = 0; u < U; ++u) {
                    const int r = (u * (DT_WARPS / 2) + w8) * per_warp + sub;
                    raw[u] = r < rows ? *reinterpret_cast<const uint4*>(w_thin + (size_t)r * n_thin + k) : make_uint4(0u, 0u, 0u, 0u);
                }
            }
            const float4 x0 = *reinterpret_cast<const float4*>(xs + k), x1 = *reinterpret_cast<const float4*>(xs + k + 4);
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const __nv_bfloat162* q = reinterpret_cast<const __nv_bfloat162*>(&raw[u]);
                const float2 w0 = __bfloat1622float2(q[0]), w1 = __bfloat1622float2(q[1]), w2 = __bfloat1622float2(q[2]),
                             w3 = __bfloat1622float2(q[3]);
                a[u] = fmaf(w0.x, x0.x, a[u]); a[u] = fmaf(w0.y, x0.y, a[u]);
                a[u] = fmaf(w1.x, x0.z, a[u]); a[u] = fmaf(w1.y, x0.w, a[u]);
                a[u] = fmaf(w2.x, x1.x, a[u]); a[u] = fmaf(w2.y, x1.y, a[u]);
                a[u] = fmaf(w3.x, x1.z, a[u]); a[u] = fmaf(w3.y, x1.w, a[u]);
            }
        }
        for (int off = L / 2; off > 0; off >>= 1)
#pragma unroll
            for (int u = 0; u < U; ++u) a[u] += __shfl_xor_sync(0xffffffffu, a[u], off);
        if (l == 0) {
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const int r = (u * (DT_WARPS / 2) + w8) * per_warp + sub;
                if (r < rows) (gates ? sgate : sg)[r] = a[u];
            }
        }
    }
    if (warp < 2) {
        const float* v = warp == 0 ? sq : sk;
        float ss = 0.f;
        for (int i = lane; i < D; i += 32) ss = fmaf(v[i], v[i], ss);
        ss = ni_warp_sum(ss);
        if (lane == 0) unit[warp] = 1.0f / sqrtf(ss + 1e-6f) * (warp == 0 ? 1.0f / sqrtf((float)D) : 1.0f);
    }
    __syncthreads();
    if (tid < D) sg[tid] = dr_decay(a_log, sg[tid] + dt);
    __syncthreads();
    const float rq = unit[0], rk = unit[1];
    float acc[VC];
#pragma unroll
    for (int j = 0; j < VC; ++j) acc[j] = 0.f;
#pragma unroll
    for (int i = 0; i < DR; ++i) {
        const int r = warp + DT_WARPS * i;
        const float gd = EXACT || r < D ? sg[r] : 0.f, kk = EXACT || r < D ? sk[r] * rk : 0.f;
#pragma unroll
        for (int j = 0; j < VC; ++j) {
            s[i][j] *= gd;
            acc[j] = fmaf(kk, s[i][j], acc[j]);
        }
    }
#pragma unroll
    for (int j = 0; j < VC; ++j) red[warp][lane + 32 * j] = acc[j];
    __syncthreads();
    if (tid < V) {                     // (V <= 128 < blockDim.x: a thread per column)
        float d = 0.f;
#pragma unroll
        for (int w = 0; w < DT_WARPS; ++w) d += red[w][tid];
        su[tid] = beta * (sv[tid] - d);
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < VC; ++j) acc[j] = 0.f;
    float u[VC];
#pragma unroll
    for (int j = 0; j < VC; ++j) u[j] = EXACT || lane + 32 * j < V ? su[lane + 32 * j] : 0.f;
#pragma unroll
    for (int i = 0; i < DR; ++i) {
        const int r = warp + DT_WARPS * i;
        const float kk = EXACT || r < D ? sk[r] * rk : 0.f, qq = EXACT || r < D ? sq[r] * rq : 0.f;
#pragma unroll
        for (int j = 0; j < VC; ++j) {
            const int col = lane + 32 * j;
            s[i][j] = fmaf(kk, u[j], s[i][j]);
            acc[j] = fmaf(qq, s[i][j], acc[j]);
            if (EXACT || (r < D && col < V)) S[(size_t)r * V + col] = s[i][j];
        }
    }
#pragma unroll
    for (int j = 0; j < VC; ++j) red[warp][lane + 32 * j] = acc[j];
    __syncthreads();
    float o = 0.f;
    if (tid < V) {
#pragma unroll
        for (int w = 0; w < DT_WARPS; ++w) o += red[w][tid];
    }
    const float ss = ni_block_sum(o * o, scratch);
    if (tid < V)
        p.y[(size_t)t * p.ld_y + (size_t)h * V + tid] =
            __float2bfloat16_rn(o * (1.0f / sqrtf(ss / (float)V + p.eps)) * norm_w * dr_sigmoid(sgate[tid]) * p.scale);
    if (taps > 1 && c >= 0 && (s_last || tid >= 2 * D)) {      // the q and k channels only by the last of the heads that share them
        if (EXACT) {
            hist[c] = h1; hist[(size_t)C + c] = h2; hist[2 * (size_t)C + c] = x;
        } else {
            for (int j = 0; j + 2 < taps; ++j) hist[(size_t)j * C + c] = hist[(size_t)(j + 1) * C + c];
            hist[(size_t)(taps - 2) * C + c] = x;
        }
    }
}

// The largest key and value sizes of ni_delta_token_step.
NI_EXPORT int ni_delta_token_max_dim() { return 128; }

// One token per request: proj FP32 [T, ld] (q | k | v from column 0, b at b_off, the thin first products - ra of the decay,
// then rg of the gate, both multiples of 8 - at thin_off), w_decay bf16 [H D, ra], w_gate bf16 [H V, rg]; y bf16, rows ld_y
// apart.  tickets: int32 zeros, at least n_seqs * G.  The state moves on, convolution history included.
NI_EXPORT int ni_delta_token_step(const float* proj, int ld, int b_off, int thin_off, const void* w_decay, int ra,
                                  const void* w_gate, int rg, const float* conv_w, const float* a_log, const float* dt_bias,
                                  const float* norm_w, float eps, float scale, float* state, long long state_stride,
                                  const int* cu_q, const int* slots, int* tickets, int n_seqs, int G, int H, int D, int V,
                                  int taps, void* y, int ld_y, cudaStream_t stream) {
    if (n_seqs <= 0) return NI_OK;
    DeltaDims dm{G, H, D, V, taps, ld, b_off, -1};
    if (int rc = dr_check(dm)) return rc;
    if (b_off < 0 || thin_off < 0 || ra <= 0 || rg <= 0 || ra % 8 || rg % 8 || ld < thin_off + ra + rg || ld_y < H * V ||
        (reinterpret_cast<size_t>(w_decay) & 15) || (reinterpret_cast<size_t>(w_gate) & 15))
        return NI_ERR_BAD_ARGUMENT;
    if (D > 128 || V > 128 || n_seqs > 65535 || ra + rg > 8192) return NI_ERR_UNSUPPORTED_SIZE;
    DeltaTokenParams p = {};
    p.proj = proj; p.w_decay = (const __nv_bfloat16*)w_decay; p.w_gate = (const __nv_bfloat16*)w_gate;
    p.conv_w = conv_w; p.a_log = a_log; p.dt_bias = dt_bias; p.norm_w = norm_w;
    p.state = state; p.state_stride = state_stride; p.cu_q = cu_q; p.slots = slots; p.tickets = tickets;
    p.y = (__nv_bfloat16*)y; p.ld_y = ld_y; p.thin_off = thin_off; p.ra = ra; p.rg = rg; p.eps = eps; p.scale = scale;
    const size_t smem = (size_t)(ra + rg) * sizeof(float);
    const bool conv_aligned = (reinterpret_cast<size_t>(conv_w) & 15) == 0;
#define GO_E(DR, VC, EXACT) delta_token_kernel<DR, VC, EXACT><<<dim3(H, n_seqs), DT_WARPS * 32, smem, stream>>>(p, dm)
#define GO(DR, VC)                                                                  \
    do {                                                                            \
        if (D == DT_WARPS * DR && V == 32 * VC && taps == 4 && conv_aligned) GO_E(DR, VC, true); \
        else GO_E(DR, VC, false);                                                   \
    } while (0)
#define GO_V(DR)                          \
    do {                                  \
        if (V <= 32) GO(DR, 1);           \
        else if (V <= 64) GO(DR, 2);      \
        else GO(DR, 4);                   \
    } while (0)
    if (D <= 32) GO_V(2);
    else if (D <= 64) GO_V(4);
    else GO_V(8);
#undef GO_V
#undef GO
#undef GO_E
    NI_RETURN_LAUNCH_STATUS();
}
