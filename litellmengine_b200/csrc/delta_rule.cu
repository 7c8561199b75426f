// The gated delta rule with a decay per key channel: per head a state S [D, V] that every token decays row by
// row, corrects towards its value and reads,
//
//     S <- diag(g_t) S        u = beta_t (v_t - S^T k_t)        S <- S + k_t u^T        o_t = S^T q_t
//
// with q and k unit vectors per head (q times D^-1/2), q, k and v behind a short causal convolution over time and
// silu, beta = sigmoid of one projection per head, g = exp(-exp(A_h) softplus(z)) with z a low-rank projection plus
// a bias, and afterwards per head o / rms(o) * w * sigmoid(a low-rank gate).  The state, the decays, the step sizes,
// the unit norms and every product of the recurrence are 32-bit CUDA-core arithmetic.
//
// The columns of S do not touch one another: column v needs k, q, g of the head and its own v_t.  So blocks take any
// number of columns of any head, and a long prompt of one request spreads over as many SMs as it has columns without
// being cut in time.  C columns (1, 2 or 4) are L lanes of a warp, each holding R = DP / L rows of all of them (rows 4 l +
// 4 L j .. + 3 of lane l), so that a vector read from shared memory serves C columns.  Along time four tokens go together.  With p_i the product of the decays of the chunk's tokens up
// to i, s_j that of the tokens behind j, and S the state that enters the chunk,
//
//     r_i = S^T (p_i k_i)     x_i = S^T (p_i q_i)                            eight products with S, one exchange of sums
//     u_i = beta_i (v_i - r_i - sum_{j<i} A_ij u_j)                           A_ij = sum_d k_i k_j (decays from j to i)
//     o_i = x_i + sum_{j<=i} B_ij u_j                                         B_ij = sum_d q_i k_j (decays from j to i)
//     S  <- p_3 S + sum_j (s_j k_j) u_j
//
// which is the recurrence with its sums regrouped: every factor is a product of decays, none is divided by one.  The
// vectors p k, p q, s k and the numbers A, B are the same for all columns of a head.
//
//   delta_prepare_kernel   a warp per (four tokens, head of q, k or v): convolution, silu, unit norm of q and k; beta
//   delta_lowrank_kernel   the second halves of both low-rank projections: decays and gates
//   delta_chunk_kernel     a warp per (four tokens, head): p k, p q, s k, p_3, A and B
//   delta_scan_kernel      one block per (entry, head, columns): the recurrence over the entry's tokens, staged sixteen
//                          at a time with cp.async into two buffers; o in 32-bit; keeps the convolutions' last inputs
//   delta_output_kernel    a warp per (token, head): norm, weight, gate, scale, store in the compute dtype
//   delta_step_kernel      all of it for entries of ONE token (decode steps): one block per (entry, head) copies the head's
//                          state and its slice of the low-rank weights into shared memory before it waits for the kernel
//                          in front of it, makes q, k, v, decays and gates, and writes the new state as it goes
//
// Per request slot the mixer keeps one row of floats: S of every head transposed, [H][V][DP] (DP = D rounded up to
// 32, 64, 128 or 256; rows from D on stay zero), then a ring of `taps` rows of the C = 2 G D + H V convolved
// projections; the row of the token at position p sits at ring row p mod taps.  A token reads the rows of positions
// p - 1 .. p - taps + 1 and writes row p mod taps, which is none of those, so in a decode step blocks that share a
// key head may read the ring while one of them writes it.
#include "common.cuh"

#define DR_TB 16            // tokens staged at a time
#define DR_CHUNK 4          // tokens that go through the state together
#define DR_LANES 8          // lanes a column of the state is spread over in the decode kernel

__device__ __forceinline__ void dr_cp16(float* smem_dst, const float* src) {
    const unsigned d = static_cast<unsigned>(__cvta_generic_to_shared(smem_dst));
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(d), "l"(src));
}

__device__ __forceinline__ void dr_prefetch(const void* p) { asm volatile("prefetch.global.L2 [%0];\n" ::"l"(p)); }

__device__ __forceinline__ float dr_silu(float x) { return __fdividef(x, 1.0f + expf(-x)); }
__device__ __forceinline__ float dr_sigmoid(float x) { return __fdividef(1.0f, 1.0f + expf(-x)); }
// ln(1 + e^x); rounding 1 + e to a float costs at most half a unit in the last place of a decay
__device__ __forceinline__ float dr_softplus(float x) { return fmaxf(x, 0.0f) + logf(1.0f + expf(-fabsf(x))); }
// the decay of one key channel: exp(-exp(A) softplus(z)); `ea` is exp(A)
__device__ __forceinline__ float dr_decay(float z, float ea) { return expf(-ea * dr_softplus(z)); }

// What the kernels know of a head's shape and of where things are.
struct DeltaShape {
    int H, G, D, V, DP, VP, taps;
    int q_off, k_off, v_off, b_off, a_off, ra, g_off, rg;      // columns of the projection; ranks of decay and gate
    long long stride;                                          // of the projection's rows
    long long slot_stride, ring_off;                           // floats of a slot; where its ring starts
};

// The convolved value of channel c (an index into q | k | v side by side, as they stand in the projection's columns
// from q_off on) for the token in batch row t: the rows of this step, then the request's ring, zeros before the start.
__device__ __forceinline__ float dr_conv(const DeltaShape& s, const float* __restrict__ proj, const float* __restrict__ w,
                                         const float* __restrict__ ring, long long t, long long row0, int pos, int c) {
    const int C = 2 * s.G * s.D + s.H * s.V;
    float acc = 0.0f;
    for (int j = 0; j < s.taps; ++j) {                          // oldest first
        const int back = s.taps - 1 - j;
        float x = 0.0f;
        if (t - back >= row0) x = proj[(t - back) * s.stride + s.q_off + c];
        else if (pos - back >= 0) x = ring[static_cast<long long>((pos - back) % s.taps) * C + c];
        acc += w[static_cast<size_t>(c) * s.taps + j] * x;
    }
    return acc;
}

#define DP_WARPS 8
#define DP_TOKENS 4
// grid: (ceil(tokens / DP_TOKENS), ceil((2 G + H) / DP_WARPS)): a warp takes four tokens of one head of q, k or v.  PER:
// channels a lane holds at a time (q and k need a whole head at once, v is taken 32 PER channels at a time).
template <int PER>
__global__ void delta_prepare_kernel(const DeltaShape s, const float* __restrict__ proj, const float* __restrict__ conv_w,
                                     const float* __restrict__ state, const int32_t* __restrict__ positions,
                                     const int32_t* __restrict__ token_entry, const int32_t* __restrict__ entry_slot,
                                     const int32_t* __restrict__ entry_q_start, float* __restrict__ qn, float* __restrict__ kn,
                                     float* __restrict__ vn, float* __restrict__ beta, int num_tokens) {
    pdl_begin();
    const int t0 = blockIdx.x * DP_TOKENS, nt = min(DP_TOKENS, num_tokens - t0);
    const int item = blockIdx.y * DP_WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (item >= 2 * s.G + s.H) return;
    const bool is_v = item >= 2 * s.G, is_q = item < s.G;
    const int head = is_v ? item - 2 * s.G : is_q ? item : item - s.G;
    const int width = is_v ? s.V : s.D, padded = is_v ? s.VP : s.DP;
    const int ch0 = is_v ? 2 * s.G * s.D + head * s.V : item * s.D;        // the head's first channel in q | k | v
    float* dst = (is_v ? vn : is_q ? qn : kn) + (static_cast<size_t>(t0) * (is_v ? s.H : s.G) + head) * padded;
    const int dst_stride = (is_v ? s.H : s.G) * padded;
    const int e0 = token_entry[t0], e3 = token_entry[t0 + nt - 1];
    // four tokens of one portion with three more of it in front of them: every input is a row of this step
    const bool plain = s.taps <= 4 && nt == DP_TOKENS && e0 == e3 && t0 - 3 >= entry_q_start[e0];
    for (int c0 = 0; c0 < padded; c0 += 32 * PER) {
        float y[DP_TOKENS][PER];
        if (plain) {
            const float* pr = proj + static_cast<long long>(t0 - 3) * s.stride + s.q_off + ch0 + c0 + lane;
#pragma unroll
            for (int i = 0; i < PER; ++i) {
                const int c = c0 + lane + 32 * i;
                if (c < width) {
                    const float* w = conv_w + static_cast<size_t>(ch0 + c) * s.taps + s.taps - 1;      // the last tap
                    const float w3 = w[0], w2 = s.taps > 1 ? w[-1] : 0.0f, w1 = s.taps > 2 ? w[-2] : 0.0f, w0 = s.taps > 3 ? w[-3] : 0.0f;
                    float x[DP_TOKENS + 3];
#pragma unroll
                    for (int j = 0; j < DP_TOKENS + 3; ++j) x[j] = pr[j * s.stride + 32 * i];
#pragma unroll
                    for (int j = 0; j < DP_TOKENS; ++j) y[j][i] = dr_silu(w0 * x[j] + w1 * x[j + 1] + w2 * x[j + 2] + w3 * x[j + 3]);
                } else {
#pragma unroll
                    for (int j = 0; j < DP_TOKENS; ++j) y[j][i] = 0.0f;
                }
            }
        } else {
#pragma unroll
            for (int j = 0; j < DP_TOKENS; ++j) {
                const int t = min(t0 + j, num_tokens - 1), e = token_entry[t];
                const float* ring = state + entry_slot[e] * s.slot_stride + s.ring_off;
#pragma unroll
                for (int i = 0; i < PER; ++i) {
                    const int c = c0 + lane + 32 * i;
                    y[j][i] = c < width ? dr_silu(dr_conv(s, proj, conv_w, ring, t, entry_q_start[e], positions[t], ch0 + c)) : 0.0f;
                }
            }
        }
        if (!is_v) {                               // unit vectors; q also times D^-1/2 (the whole head is here: D <= 32 PER)
            float n[DP_TOKENS];
#pragma unroll
            for (int j = 0; j < DP_TOKENS; ++j) {
                n[j] = 0.0f;
#pragma unroll
                for (int i = 0; i < PER; ++i) n[j] += y[j][i] * y[j][i];
            }
#pragma unroll
            for (int m = 16; m > 0; m >>= 1)
#pragma unroll
                for (int j = 0; j < DP_TOKENS; ++j) n[j] += __shfl_xor_sync(0xffffffffu, n[j], m);
#pragma unroll
            for (int j = 0; j < DP_TOKENS; ++j) {
                const float inv = 1.0f / sqrtf((n[j] + 1e-6f) * (is_q ? static_cast<float>(s.D) : 1.0f));
#pragma unroll
                for (int i = 0; i < PER; ++i) y[j][i] *= inv;
            }
        }
#pragma unroll
        for (int j = 0; j < DP_TOKENS; ++j)
#pragma unroll
            for (int i = 0; i < PER; ++i) {
                const int c = c0 + lane + 32 * i;
                if (j < nt && c < padded) dst[j * dst_stride + c] = y[j][i];      // behind a head's end: zeros
            }
    }
    if (is_v && lane < nt) beta[static_cast<size_t>(t0 + lane) * s.H + head] = dr_sigmoid(proj[(t0 + lane) * s.stride + s.b_off + head]);
}

// Second halves of the low-rank projections.  A block takes DL_TOKENS tokens and DL_CHANNELS channels (two a thread) of
// either the decays or the gates; the tokens' first halves sit in shared memory as [rank][tokens], so that a thread
// reads four tokens' values at a time and each weight serves all of the block's tokens.  Weights are transposed,
// [rank][channels].
#define DL_TOKENS 16
#define DL_PITCH 20               // floats from rank to rank in shared memory
#define DL_THREADS 128
#define DL_CHANNELS (2 * DL_THREADS)
template <typename TW>
__global__ void __launch_bounds__(DL_THREADS) delta_lowrank_kernel(
    const DeltaShape s, const float* __restrict__ proj, const TW* __restrict__ wa, const float* __restrict__ dt_bias,
    const float* __restrict__ a_log, const TW* __restrict__ wg, float* __restrict__ decay, float* __restrict__ gate, int num_tokens,
    int decay_blocks) {
    pdl_begin();
    extern __shared__ __align__(16) float a[];
    const bool is_decay = static_cast<int>(blockIdx.y) < decay_blocks;
    const int rank = is_decay ? s.ra : s.rg, off = is_decay ? s.a_off : s.g_off;
    const int channels = is_decay ? s.H * s.D : s.H * s.V;
    const TW* w = is_decay ? wa : wg;
    const int t0 = blockIdx.x * DL_TOKENS;
    const int nt = min(DL_TOKENS, num_tokens - t0);
    for (int idx = threadIdx.x; idx < DL_TOKENS * rank; idx += blockDim.x) {
        const int t = idx / rank, j = idx - t * rank;
        a[j * DL_PITCH + t] = t < nt ? proj[static_cast<size_t>(t0 + t) * s.stride + off + j] : 0.0f;
    }
    __syncthreads();
    const int c0 = (is_decay ? blockIdx.y : blockIdx.y - decay_blocks) * DL_CHANNELS + threadIdx.x;
    const bool there[2] = {c0 < channels, c0 + DL_THREADS < channels};
    if (!there[0]) return;
    float z[2][DL_TOKENS];
#pragma unroll
    for (int n = 0; n < 2; ++n) {
        const float bias = is_decay && there[n] ? dt_bias[c0 + n * DL_THREADS] : 0.0f;
#pragma unroll
        for (int t = 0; t < DL_TOKENS; ++t) z[n][t] = bias;
    }
    for (int j0 = 0; j0 < rank; j0 += 4) {                      // eight weights in flight
        float wv[2][4];
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int u = 0; u < 4; ++u)
                wv[n][u] = j0 + u < rank && there[n] ? to_f32(w[static_cast<size_t>(j0 + u) * channels + c0 + n * DL_THREADS]) : 0.0f;
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const float4* ar = reinterpret_cast<const float4*>(a + min(j0 + u, rank - 1) * DL_PITCH);
#pragma unroll
            for (int t = 0; t < DL_TOKENS; t += 4) {
                const float4 v = ar[t >> 2];
#pragma unroll
                for (int n = 0; n < 2; ++n) {
                    z[n][t] += wv[n][u] * v.x;
                    z[n][t + 1] += wv[n][u] * v.y;
                    z[n][t + 2] += wv[n][u] * v.z;
                    z[n][t + 3] += wv[n][u] * v.w;
                }
            }
        }
    }
#pragma unroll
    for (int n = 0; n < 2; ++n) {
        if (!there[n]) continue;
        const int c = c0 + n * DL_THREADS;
        if (is_decay) {
            const int h = c / s.D, d = c - h * s.D;
            const float ea = expf(a_log[h]);
#pragma unroll
            for (int t = 0; t < DL_TOKENS; ++t)
                if (t < nt) decay[(static_cast<size_t>(t0 + t) * s.H + h) * s.DP + d] = dr_decay(z[n][t], ea);
        } else {
#pragma unroll
            for (int t = 0; t < DL_TOKENS; ++t)
                if (t < nt) gate[static_cast<size_t>(t0 + t) * channels + c] = dr_sigmoid(z[n][t]);
        }
    }
}

// Sum over the eight lanes of a column.
__device__ __forceinline__ float dr_lane_sum(float v) {
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    v += __shfl_xor_sync(0xffffffffu, v, 2);
    v += __shfl_xor_sync(0xffffffffu, v, 4);
    return v;
}

// One token against the R rows (R / 4 groups of four) that a lane holds of a column: decays S, returns o and writes.
template <int R>
__device__ __forceinline__ float dr_token(float (&S)[R], const float* __restrict__ k, const float* __restrict__ q,
                                          const float* __restrict__ g, int l, float v, float beta, float kq) {
    float4 kk[R / 4];
    float r0 = 0.0f, r1 = 0.0f, o0 = 0.0f, o1 = 0.0f;
#pragma unroll
    for (int j = 0; j < R / 4; ++j) {
        const float4 gg = *reinterpret_cast<const float4*>(g + 4 * l + 32 * j);
        const float4 qq = *reinterpret_cast<const float4*>(q + 4 * l + 32 * j);
        kk[j] = *reinterpret_cast<const float4*>(k + 4 * l + 32 * j);
        S[4 * j] *= gg.x;
        S[4 * j + 1] *= gg.y;
        S[4 * j + 2] *= gg.z;
        S[4 * j + 3] *= gg.w;
        r0 += S[4 * j] * kk[j].x;
        r1 += S[4 * j + 1] * kk[j].y;
        r0 += S[4 * j + 2] * kk[j].z;
        r1 += S[4 * j + 3] * kk[j].w;
        o0 += S[4 * j] * qq.x;
        o1 += S[4 * j + 1] * qq.y;
        o0 += S[4 * j + 2] * qq.z;
        o1 += S[4 * j + 3] * qq.w;
    }
    const float r = dr_lane_sum(r0 + r1), o = dr_lane_sum(o0 + o1);
    const float u = beta * (v - r);
#pragma unroll
    for (int j = 0; j < R / 4; ++j) {
        S[4 * j] += kk[j].x * u;
        S[4 * j + 1] += kk[j].y * u;
        S[4 * j + 2] += kk[j].z * u;
        S[4 * j + 3] += kk[j].w * u;
    }
    return o + kq * u;
}

// One level of a sum over lanes that also deals the values out: of N values each lane keeps the N / 2 that its bit
// `MASK` says, summed with its partner's.
template <int N, int MASK>
__device__ __forceinline__ void dr_deal(float* v, int lane) {
    const bool up = lane & MASK;
#pragma unroll
    for (int n = 0; n < N / 2; ++n) {
        const float send = up ? v[n] : v[n + N / 2], keep = up ? v[n + N / 2] : v[n];
        v[n] = keep + __shfl_xor_sync(0xffffffffu, send, MASK);
    }
}

// Sums of NV values over the L lanes of a group, left in sums[0 .. NV - 1] (in shared memory).
template <int NV, int L>
__device__ __forceinline__ void dr_sums(float (&v)[NV], int lane, int l, float* sums) {
    if constexpr (NV > 1 && L >= 2) dr_deal<NV, L / 2>(v, lane);
    if constexpr (NV > 2 && L >= 4) dr_deal<NV / 2, L / 4>(v, lane);
    if constexpr (NV > 4 && L >= 8) dr_deal<NV / 4, L / 8>(v, lane);
    if constexpr (NV > 8 && L >= 16) dr_deal<NV / 8, L / 16>(v, lane);
    if constexpr (NV > 16 && L >= 32) dr_deal<NV / 16, L / 32>(v, lane);
    constexpr int REST = NV >= L ? 1 : L / NV, K = NV >= L ? NV / L : 1;       // lanes that share a value; values a lane holds
#pragma unroll
    for (int m = REST / 2; m > 0; m >>= 1) v[0] += __shfl_xor_sync(0xffffffffu, v[0], m);
    if (NV >= L || (l & (REST - 1)) == 0) {
#pragma unroll
        for (int n = 0; n < K; ++n) sums[(l / REST) * K + n] = v[n];
    }
}

#define DR_NUM 24                             // numbers a chunk: A (six, two unused), then B as [4][4], zero above its diagonal

// Where a chunk's shared vectors and numbers are: chunks start at every fourth row of an entry, so row / 4 + entry is a
// number of its own for each of them.
__device__ __forceinline__ long long dr_chunk_place(long long row, int entry) { return row / DR_CHUNK + entry; }

// What a chunk's four tokens share over all columns of a head: a warp per (first token of a chunk, head); tokens that
// begin no chunk have no work.  pk = p k, pq = p q, and in place of the decays s k; total = p_3; num = A and B.
#define DC_WARPS 4
template <int DP>
__global__ void __launch_bounds__(DC_WARPS * 32) delta_chunk_kernel(
    const DeltaShape s, const float* __restrict__ qn, const float* __restrict__ kn, float* decay, float* __restrict__ pk,
    float* __restrict__ pq, float* __restrict__ total, float* __restrict__ num, const int32_t* __restrict__ token_entry,
    const int32_t* __restrict__ entry_q_start, const int32_t* __restrict__ entry_q_len, int num_tokens) {
    // no early invitation: the blocks of the scan behind this kernel would be dealt to whichever SMs have room while
    // this one drains, several to one SM, and the scan takes as long as its fullest SM
    pdl_wait();
    const long long t = blockIdx.x;
    const int h = blockIdx.y * DC_WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (h >= s.H) return;
    const int entry = token_entry[t];
    const long long row0 = entry_q_start[entry];
    if ((t - row0) % DR_CHUNK) return;
    const int nt = static_cast<int>(min(static_cast<long long>(DR_CHUNK), row0 + entry_q_len[entry] - t));
    const int kvh = h / (s.H / s.G);
    const size_t place = static_cast<size_t>(dr_chunk_place(t, entry)) * s.H + h;
    float acc[16];                            // A10 A20 A21 A30 A31 A32, then B00 B10 B11 B20 B21 B22 B30 B31 B32 B33
#pragma unroll
    for (int n = 0; n < 16; ++n) acc[n] = 0.0f;
    for (int x = lane * 4; x < DP; x += 128) {
        float kk[4][4], qq[4][4], gg[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            float4 a = make_float4(0, 0, 0, 0), b = a, c = make_float4(1, 1, 1, 1);      // a missing token
            if (i < nt) {
                const size_t at = (static_cast<size_t>(t + i) * s.G + kvh) * DP + x;
                a = *reinterpret_cast<const float4*>(kn + at);
                b = *reinterpret_cast<const float4*>(qn + at);
                c = *reinterpret_cast<const float4*>(decay + (static_cast<size_t>(t + i) * s.H + h) * DP + x);
            }
            kk[i][0] = a.x; kk[i][1] = a.y; kk[i][2] = a.z; kk[i][3] = a.w;
            qq[i][0] = b.x; qq[i][1] = b.y; qq[i][2] = b.z; qq[i][3] = b.w;
            gg[i][0] = c.x; gg[i][1] = c.y; gg[i][2] = c.z; gg[i][3] = c.w;
        }
        float sk[4][4], p[4] = {1.0f, 1.0f, 1.0f, 1.0f};
#pragma unroll
        for (int e = 0; e < 4; ++e)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                float w = kk[j][e];
                acc[6 + j * (j + 1) / 2 + j] += qq[j][e] * w;
#pragma unroll
                for (int i = j + 1; i < 4; ++i) {
                    w *= gg[i][e];
                    acc[i * (i - 1) / 2 + j] += kk[i][e] * w;
                    acc[6 + i * (i + 1) / 2 + j] += qq[i][e] * w;
                }
                sk[j][e] = w;
            }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
#pragma unroll
            for (int e = 0; e < 4; ++e) p[e] *= gg[i][e];
            if (i < nt) {
                const size_t at = (static_cast<size_t>(t + i) * s.H + h) * DP + x;
                *reinterpret_cast<float4*>(pk + at) = make_float4(p[0] * kk[i][0], p[1] * kk[i][1], p[2] * kk[i][2], p[3] * kk[i][3]);
                *reinterpret_cast<float4*>(pq + at) = make_float4(p[0] * qq[i][0], p[1] * qq[i][1], p[2] * qq[i][2], p[3] * qq[i][3]);
                *reinterpret_cast<float4*>(decay + at) = make_float4(sk[i][0], sk[i][1], sk[i][2], sk[i][3]);
            }
        }
        *reinterpret_cast<float4*>(total + place * DP + x) = make_float4(p[0], p[1], p[2], p[3]);
    }
    dr_deal<16, 16>(acc, lane);
    dr_deal<8, 8>(acc, lane);
    dr_deal<4, 4>(acc, lane);
    dr_deal<2, 2>(acc, lane);
    const float sum = acc[0] + __shfl_xor_sync(0xffffffffu, acc[0], 1);
    const int n = lane >> 1;                  // the value this pair of lanes holds
    float* out = num + place * DR_NUM;
    if (lane & 1) {                           // the odd lanes clear what is above B's diagonal
        if (n < 4)
            for (int j = n + 1; j < 4; ++j) out[8 + 4 * n + j] = 0.0f;
    } else if (n < 6) {
        out[n] = sum;
    } else {
        const int m = n - 6, i = m < 1 ? 0 : m < 3 ? 1 : m < 6 ? 2 : 3;
        out[8 + 4 * i + (m - i * (i + 1) / 2)] = sum;
    }
}

// grid (entries, H, column tiles): WARPS warps a block, each 32 / L groups of C columns.
template <int DP, int C, int WARPS>
__global__ void __launch_bounds__(WARPS * 32) delta_scan_kernel(
    const DeltaShape s, const float* __restrict__ proj, const float* __restrict__ pq, const float* __restrict__ pk,
    const float* __restrict__ vn, const float* __restrict__ beta, const float* __restrict__ sk, const float* __restrict__ total,
    const float* __restrict__ num, float* __restrict__ o, float* __restrict__ state, const int32_t* __restrict__ positions,
    const int32_t* __restrict__ entry_slot, const int32_t* __restrict__ entry_q_start, const int32_t* __restrict__ entry_q_len) {
    pdl_begin();
    constexpr int L = DP >= 128 ? 32 : DP / 4, R = DP / L, THREADS = WARPS * 32, CHUNKS = DR_TB / DR_CHUNK;
    constexpr int COLS = WARPS * (32 / L) * C, NV = 8 * C;
    // a buffer: q, k, s k, v of a batch of tokens, then beta; then p_3 and the numbers of its chunks
    constexpr int BUF = DR_TB * (3 * DP + COLS + 1) + CHUNKS * (DP + DR_NUM);
    extern __shared__ __align__(16) float smem[];
    const int entry = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31;
    const int c0 = blockIdx.z * COLS;
    const int l = lane & (L - 1), group = tid / L, cb = group * C;          // the group's first column in the block
    float* sums = smem + 2 * BUF + group * NV;                  // [8][C]: the group's sums, by value and column
    const long long row0 = entry_q_start[entry];
    const int count = entry_q_len[entry];
    float* slot = state + entry_slot[entry] * s.slot_stride;
    float* col_state = slot + (static_cast<long long>(h) * s.V + c0 + cb) * DP + 4 * l;
    const int cols_here = s.V - c0 - cb;                        // columns of the group that exist, if fewer than C
    float S[C][R];
#pragma unroll
    for (int m = 0; m < C; ++m)
#pragma unroll
        for (int j = 0; j < R / 4; ++j) {
            const float4 x = m < cols_here ? *reinterpret_cast<const float4*>(col_state + m * DP + 4 * L * j) : make_float4(0, 0, 0, 0);
            S[m][4 * j] = x.x; S[m][4 * j + 1] = x.y; S[m][4 * j + 2] = x.z; S[m][4 * j + 3] = x.w;
        }
    const size_t first = (static_cast<size_t>(row0) * s.H + h) * DP;
    const int row_stride = s.H * DP;
    const size_t place = static_cast<size_t>(dr_chunk_place(row0, entry)) * s.H + h;
    auto stage = [&](int done, int buf) {
        constexpr int PIECES = DP / 4, STEP = THREADS / PIECES > 0 ? THREADS / PIECES : 1;
        const int nb = min(DR_TB, count - done);
        float* bq = smem + buf * BUF;
        float* bk = bq + DR_TB * DP;
        float* bs = bk + DR_TB * DP;
        float* bv = bs + DR_TB * DP;
        float* bb = bv + DR_TB * COLS;
        float* bt = bb + DR_TB;
        float* bn = bt + CHUNKS * DP;
        const size_t at = first + static_cast<size_t>(done) * row_stride;
        for (int x = (tid % PIECES) * 4; x < DP; x += THREADS * 4)
            for (int tok = tid / PIECES; tok < nb; tok += STEP) {
                const size_t from = at + static_cast<size_t>(tok) * row_stride + x;
                dr_cp16(bq + tok * DP + x, pq + from);
                dr_cp16(bk + tok * DP + x, pk + from);
                dr_cp16(bs + tok * DP + x, sk + from);
            }
        const int chunks = (nb + DR_CHUNK - 1) / DR_CHUNK;
        const size_t first_chunk = place + static_cast<size_t>(done / DR_CHUNK) * s.H;
        for (int idx = tid; idx < chunks * PIECES; idx += THREADS) {
            const int ch = idx / PIECES, x = (idx - ch * PIECES) * 4;
            dr_cp16(bt + ch * DP + x, total + (first_chunk + static_cast<size_t>(ch) * s.H) * DP + x);
        }
        for (int idx = tid; idx < chunks * (DR_NUM / 4); idx += THREADS) {
            const int ch = idx / (DR_NUM / 4), x = (idx - ch * (DR_NUM / 4)) * 4;
            dr_cp16(bn + ch * DR_NUM + x, num + (first_chunk + static_cast<size_t>(ch) * s.H) * DR_NUM + x);
        }
        for (int idx = tid; idx < nb * (COLS / 4); idx += THREADS) {
            const int tok = idx / (COLS / 4), x = (idx - tok * (COLS / 4)) * 4;
            if (c0 + x < s.VP) dr_cp16(bv + tok * COLS + x, vn + (static_cast<size_t>(row0 + done + tok) * s.H + h) * s.VP + c0 + x);
        }
        if (tid < nb) {
            const unsigned d = static_cast<unsigned>(__cvta_generic_to_shared(bb + tid));
            asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(d), "l"(beta + static_cast<size_t>(row0 + done + tid) * s.H + h));
        }
        for (int idx = nb * DP + tid; idx < chunks * DR_CHUNK * DP; idx += THREADS) bs[idx] = 0.0f;      // missing tokens write nothing
        asm volatile("cp.async.commit_group;\n" ::);
    };
    stage(0, 0);
    for (int done = 0, b = 0; done < count; done += DR_TB, ++b) {
        const int nb = min(DR_TB, count - done);
        if (done + DR_TB < count) {
            stage(done + DR_TB, (b + 1) & 1);
            asm volatile("cp.async.wait_group 1;\n" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        }
        __syncthreads();
        const float* bq = smem + (b & 1) * BUF;
        const float* bk = bq + DR_TB * DP;
        const float* bs = bk + DR_TB * DP;
        const float* bv = bs + DR_TB * DP;
        const float* bb = bv + DR_TB * COLS;
        const float* bt = bb + DR_TB;
        const float* bn = bt + CHUNKS * DP;
        const int chunks = (nb + DR_CHUNK - 1) / DR_CHUNK;
        for (int ch = 0; ch < chunks; ++ch) {
            const float* k = bk + ch * 4 * DP + 4 * l;
            const float* q = bq + ch * 4 * DP + 4 * l;
            const float* w = bs + ch * 4 * DP + 4 * l;
            float v[NV];                      // value n of column m at n C + m: r_0 .. r_3, x_0 .. x_3
#pragma unroll
            for (int n = 0; n < NV; ++n) v[n] = 0.0f;
#pragma unroll
            for (int j = 0; j < R / 4; ++j)
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const float4 a = *reinterpret_cast<const float4*>(k + i * DP + 4 * L * j);
                    const float4 e = *reinterpret_cast<const float4*>(q + i * DP + 4 * L * j);
#pragma unroll
                    for (int m = 0; m < C; ++m) {
                        v[i * C + m] += S[m][4 * j] * a.x;
                        v[(4 + i) * C + m] += S[m][4 * j] * e.x;
                        v[i * C + m] += S[m][4 * j + 1] * a.y;
                        v[(4 + i) * C + m] += S[m][4 * j + 1] * e.y;
                        v[i * C + m] += S[m][4 * j + 2] * a.z;
                        v[(4 + i) * C + m] += S[m][4 * j + 2] * e.z;
                        v[i * C + m] += S[m][4 * j + 3] * a.w;
                        v[(4 + i) * C + m] += S[m][4 * j + 3] * e.w;
                    }
                }
            dr_sums<NV, L>(v, lane, l, sums);
            __syncwarp();
            const float* nu = bn + ch * DR_NUM;
            const float4 a0 = *reinterpret_cast<const float4*>(nu), be = *reinterpret_cast<const float4*>(bb + ch * 4);
            const float2 a1 = *reinterpret_cast<const float2*>(nu + 4);
            const int left = nb - ch * DR_CHUNK;               // tokens of the chunk; the missing ones write nothing
            float u[4][C];
#pragma unroll
            for (int m = 0; m < C; ++m) {
                const float* vt = bv + ch * 4 * COLS + cb + m;
                u[0][m] = be.x * (vt[0] - sums[m]);
                u[1][m] = left > 1 ? be.y * (vt[COLS] - sums[C + m] - a0.x * u[0][m]) : 0.0f;
                u[2][m] = left > 2 ? be.z * (vt[2 * COLS] - sums[2 * C + m] - a0.y * u[0][m] - a0.z * u[1][m]) : 0.0f;
                u[3][m] = left > 3 ? be.w * (vt[3 * COLS] - sums[3 * C + m] - a0.w * u[0][m] - a1.x * u[1][m] - a1.y * u[2][m]) : 0.0f;
            }
#pragma unroll
            for (int n = l; n < 4 * C; n += L) {                // token n / C of column n % C
                const int i = n / C, m = n % C;
                const float4 bi = *reinterpret_cast<const float4*>(nu + 8 + 4 * i);
                float um[4];
#pragma unroll
                for (int t = 0; t < 4; ++t)
                    um[t] = C == 1 ? u[t][0] : C == 2 ? ((m & 1) ? u[t][C - 1] : u[t][0])
                                             : (m & 2) ? ((m & 1) ? u[t][C - 1] : u[t][C >= 4 ? 2 : 0]) : ((m & 1) ? u[t][C >= 2 ? 1 : 0] : u[t][0]);
                const float out = sums[(4 + i) * C + m] + bi.x * um[0] + bi.y * um[1] + bi.z * um[2] + bi.w * um[3];
                if (i < left && m < cols_here)
                    o[(static_cast<size_t>(row0 + done + ch * DR_CHUNK + i) * s.H + h) * s.V + c0 + cb + m] = out;
            }
#pragma unroll
            for (int j = 0; j < R / 4; ++j) {
                const float4 p = *reinterpret_cast<const float4*>(bt + ch * DP + 4 * l + 4 * L * j);
                const float4 w0 = *reinterpret_cast<const float4*>(w + 4 * L * j), w1 = *reinterpret_cast<const float4*>(w + DP + 4 * L * j),
                             w2 = *reinterpret_cast<const float4*>(w + 2 * DP + 4 * L * j),
                             w3 = *reinterpret_cast<const float4*>(w + 3 * DP + 4 * L * j);
#pragma unroll
                for (int m = 0; m < C; ++m) {
                    S[m][4 * j] = p.x * S[m][4 * j] + w0.x * u[0][m] + w1.x * u[1][m] + w2.x * u[2][m] + w3.x * u[3][m];
                    S[m][4 * j + 1] = p.y * S[m][4 * j + 1] + w0.y * u[0][m] + w1.y * u[1][m] + w2.y * u[2][m] + w3.y * u[3][m];
                    S[m][4 * j + 2] = p.z * S[m][4 * j + 2] + w0.z * u[0][m] + w1.z * u[1][m] + w2.z * u[2][m] + w3.z * u[3][m];
                    S[m][4 * j + 3] = p.w * S[m][4 * j + 3] + w0.w * u[0][m] + w1.w * u[1][m] + w2.w * u[2][m] + w3.w * u[3][m];
                }
            }
            __syncwarp();                                       // `sums` is written again
        }
        __syncthreads();                      // this buffer is filled again two batches on
    }
#pragma unroll
    for (int m = 0; m < C; ++m)
        if (m < cols_here)
#pragma unroll
            for (int j = 0; j < R / 4; ++j)
                *reinterpret_cast<float4*>(col_state + m * DP + 4 * L * j) = make_float4(S[m][4 * j], S[m][4 * j + 1], S[m][4 * j + 2], S[m][4 * j + 3]);
    // the convolutions' inputs of the portion's last tokens (the kernels before this one have read the ring)
    const int channels = 2 * s.G * s.D + s.H * s.V, keep = min(count, s.taps - 1), kvh = h / (s.H / s.G);
    float* ring = slot + s.ring_off;
    const bool with_qk = blockIdx.z == 0 && h % (s.H / s.G) == 0;
    for (int i = 0; i < keep; ++i) {
        const long long t = row0 + count - keep + i;
        float* dst = ring + static_cast<long long>(positions[t] % s.taps) * channels;
        const float* src = proj + t * s.stride + s.q_off;
        if (with_qk)
            for (int d = tid; d < s.D; d += THREADS) {
                dst[kvh * s.D + d] = src[kvh * s.D + d];
                dst[(s.G + kvh) * s.D + d] = src[(s.G + kvh) * s.D + d];
            }
        for (int x = tid; x < COLS && c0 + x < s.V; x += THREADS) {
            const int ch = 2 * s.G * s.D + h * s.V + c0 + x;
            dst[ch] = src[ch];
        }
    }
}

// A warp per (token, head): o / rms(o) * w * gate * scale.
template <typename TO>
__global__ void delta_output_kernel(const float* __restrict__ o, const float* __restrict__ gate, const float* __restrict__ norm_w,
                                    float eps, float out_scale, TO* __restrict__ out, long long out_stride, int out_off, int H,
                                    int V, long long items) {
    pdl_begin();
    const long long item = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (item >= items) return;
    const int lane = threadIdx.x & 31;
    const long long t = item / H;
    const int h = static_cast<int>(item - t * H);
    const float* row = o + item * V;
    const float* gr = gate + item * V;
    float ss = 0.0f;
    for (int c = lane; c < V; c += 32) ss += row[c] * row[c];
    ss = warp_sum(ss);
    const float inv = 1.0f / sqrtf(ss / static_cast<float>(V) + eps);
    TO* orow = out + t * out_stride + out_off + h * V;
    for (int c = lane; c < V; c += 32) orow[c] = from_f32<TO>(row[c] * inv * norm_w[c] * gr[c] * out_scale);
}

// Entries that bring one token: one block per (entry, head).  STAGED: the head's state (V columns of DP floats) and, with
// `low_staged`, its slices of the low-rank weights are copied into shared memory before the block waits for the kernel in
// front of it (nothing else in a step writes this stage's states, and the weights never change); otherwise they are read
// as they are needed.
template <int R, typename TW, typename TO, bool STAGED>
__global__ void __launch_bounds__(512) delta_step_kernel(
    const DeltaShape s, const float* __restrict__ proj, const float* __restrict__ conv_w, const TW* __restrict__ wa,
    const float* __restrict__ dt_bias, const float* __restrict__ a_log, const TW* __restrict__ wg,
    const float* __restrict__ norm_w, float eps, float out_scale, TO* __restrict__ out, long long out_stride, int out_off,
    float* __restrict__ state, const int32_t* __restrict__ positions, const int32_t* __restrict__ entry_slot,
    const int32_t* __restrict__ entry_q_start, int low_staged) {
    pdl_invite();
    constexpr int DP = DR_LANES * R;
    extern __shared__ __align__(16) float smem[];
    float* sq = smem;                         // [DP] each
    float* sk = sq + DP;
    float* sg = sk + DP;
    float* red = sg + DP;                     // 36
    float* sv = red + 36;                     // [V] each
    float* so = sv + s.V;
    float* sgate = so + s.V;
    float* first = sgate + s.V;               // [ra + rg]: the first halves of the low-rank projections
    const int chans = s.D + s.V, tid = threadIdx.x, nthreads = blockDim.x;
    int parts = nthreads / chans;             // threads that share a channel's low-rank sum
    parts = parts < 1 ? 1 : parts > 8 ? 8 : parts;
    float* split = first + s.ra + s.rg;       // [parts][D + V]
    float* held = smem + ((3 * DP + 36 + 3 * s.V + s.ra + s.rg + parts * chans + 3) & ~3);     // STAGED: [V][DP]
    TW* low = reinterpret_cast<TW*>(held + (STAGED ? static_cast<size_t>(s.V) * DP : 0));      // STAGED: [ra][D], [rg][V]
    const int entry = blockIdx.x, h = blockIdx.y;
    const int kvh = h / (s.H / s.G);
    const long long t = entry_q_start[entry];
    const int pos = positions[t];
    float* slot = state + entry_slot[entry] * s.slot_stride;
    float* head_state = slot + static_cast<long long>(h) * s.V * DP;
    float* ring = slot + s.ring_off;
    const int C = 2 * s.G * s.D + s.H * s.V;
    // what the block will read of weights and of earlier steps' inputs, on its way to the cache before the wait
    const int cq = kvh * s.D, ck = (s.G + kvh) * s.D, cv = 2 * s.G * s.D + h * s.V;
    for (int i = tid * 32; i < s.D * s.taps; i += nthreads * 32) {
        dr_prefetch(conv_w + static_cast<size_t>(cq) * s.taps + i);
        dr_prefetch(conv_w + static_cast<size_t>(ck) * s.taps + i);
    }
    for (int i = tid * 32; i < s.V * s.taps; i += nthreads * 32) dr_prefetch(conv_w + static_cast<size_t>(cv) * s.taps + i);
    for (int i = tid; i < s.taps * 32; i += nthreads) {         // a ring row's three pieces in lines of 32 floats
        const float* row = ring + static_cast<long long>(i >> 5) * C;
        for (int x = (i & 31) * 32; x < s.D; x += 1024) {
            dr_prefetch(row + cq + x);
            dr_prefetch(row + ck + x);
        }
        for (int x = (i & 31) * 32; x < s.V; x += 1024) dr_prefetch(row + cv + x);
    }
    for (int i = tid * 32; i < s.D; i += nthreads * 32) dr_prefetch(dt_bias + h * s.D + i);
    for (int i = tid * 32; i < s.V; i += nthreads * 32) dr_prefetch(norm_w + i);
    if (!(STAGED && low_staged)) {
        for (int i = tid; i < s.ra; i += nthreads)
            for (int x = 0; x < s.D; x += 128 / static_cast<int>(sizeof(TW))) dr_prefetch(wa + static_cast<size_t>(i) * s.H * s.D + h * s.D + x);
        for (int i = tid; i < s.rg; i += nthreads)
            for (int x = 0; x < s.V; x += 128 / static_cast<int>(sizeof(TW))) dr_prefetch(wg + static_cast<size_t>(i) * s.H * s.V + h * s.V + x);
    }
    const float ea = expf(a_log[h]);
    if (STAGED) {
        constexpr int PER = 16 / sizeof(TW);
        const int na = low_staged ? s.ra * (s.D / PER) : 0, ng = low_staged ? s.rg * (s.V / PER) : 0;
        for (int i = tid; i < na + ng; i += nthreads) {
            const bool is_decay = i < na;
            const int n = is_decay ? i : i - na, w = is_decay ? s.D : s.V, j = n / (w / PER), x = (n - j * (w / PER)) * PER;
            const TW* src = is_decay ? wa + static_cast<size_t>(j) * s.H * s.D + h * s.D + x : wg + static_cast<size_t>(j) * s.H * s.V + h * s.V + x;
            dr_cp16(reinterpret_cast<float*>(low + (is_decay ? 0 : s.ra * s.D) + j * w + x), reinterpret_cast<const float*>(src));
        }
        for (int i = tid * 4; i < s.V * DP; i += nthreads * 4) dr_cp16(held + i, head_state + i);
        asm volatile("cp.async.commit_group;\n" ::);
    }
    pdl_wait();
    const float* pr = proj + t * s.stride;
    const float beta = dr_sigmoid(pr[s.b_off + h]);
    for (int j = tid; j < s.ra + s.rg; j += nthreads) first[j] = j < s.ra ? pr[s.a_off + j] : pr[s.g_off + j - s.ra];
    // convolutions; the row's own place in the ring is none that any block reads in this step
    float* mine = ring + static_cast<long long>(pos % s.taps) * C;
    const bool with_qk = h % (s.H / s.G) == 0;
    for (int i = tid; i < 2 * DP + s.V; i += nthreads) {
        if (i < 2 * DP) {
            const int d = i < DP ? i : i - DP;
            float x = 0.0f;
            if (d < s.D) {
                const int ch = (i < DP ? kvh : s.G + kvh) * s.D + d;
                x = dr_silu(dr_conv(s, proj, conv_w, ring, t, t, pos, ch));
                if (with_qk && s.taps > 1) mine[ch] = pr[s.q_off + ch];
            }
            sq[i] = x;                        // q, then k behind it
        } else {
            const int ch = 2 * s.G * s.D + h * s.V + (i - 2 * DP);
            sv[i - 2 * DP] = dr_silu(dr_conv(s, proj, conv_w, ring, t, t, pos, ch));
            if (s.taps > 1) mine[ch] = pr[s.q_off + ch];
        }
    }
    if (STAGED) asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    __syncthreads();
    for (int i = tid; i < parts * chans; i += nthreads) {       // low-rank second halves
        const int p = i / chans, ch = i - p * chans;
        const bool is_decay = ch < s.D;
        const int rank = is_decay ? s.ra : s.rg, x = is_decay ? ch : ch - s.D;
        const bool here = STAGED && low_staged;
        const int width = here ? (is_decay ? s.D : s.V) : (is_decay ? s.H * s.D : s.H * s.V);
        const TW* w = here ? low + (is_decay ? 0 : s.ra * s.D) + x : is_decay ? wa + h * s.D + x : wg + h * s.V + x;
        const float* a = is_decay ? first : first + s.ra;
        const int per = (rank + parts - 1) / parts, j1 = min(rank, (p + 1) * per);
        float z = 0.0f;
        int j = p * per;
        for (; j + 16 <= j1; j += 16) {
            float wv[16];
#pragma unroll
            for (int u = 0; u < 16; ++u) wv[u] = to_f32(w[(j + u) * width]);
#pragma unroll
            for (int u = 0; u < 16; ++u) z += wv[u] * a[j + u];
        }
        for (; j < j1; ++j) z += to_f32(w[j * width]) * a[j];
        split[i] = z;
    }
    const int warp = tid >> 5, lane = tid & 31;
    if (warp == 0) {                          // unit norms and k . q
        float qq = 0.0f, kk = 0.0f, qk = 0.0f;
        for (int d = lane; d < DP; d += 32) {
            qq += sq[d] * sq[d];
            kk += sk[d] * sk[d];
            qk += sq[d] * sk[d];
        }
        qq = warp_sum(qq);
        kk = warp_sum(kk);
        qk = warp_sum(qk);
        const float iq = 1.0f / sqrtf(qq + 1e-6f) / sqrtf(static_cast<float>(s.D)), ik = 1.0f / sqrtf(kk + 1e-6f);
        for (int d = lane; d < DP; d += 32) {
            sq[d] *= iq;
            sk[d] *= ik;
        }
        if (lane == 0) red[33] = qk * iq * ik;
    }
    __syncthreads();
    for (int i = tid; i < DP + s.V; i += nthreads) {
        if (i < DP) {
            float g = 0.0f;
            if (i < s.D) {
                float z = dt_bias[h * s.D + i];
                for (int p = 0; p < parts; ++p) z += split[p * chans + i];
                g = dr_decay(z, ea);
            }
            sg[i] = g;
        } else {
            float z = 0.0f;
            for (int p = 0; p < parts; ++p) z += split[p * chans + s.D + (i - DP)];
            sgate[i - DP] = dr_sigmoid(z);
        }
    }
    __syncthreads();
    const float kq = red[33];
    const int l = tid & (DR_LANES - 1), cols = nthreads / DR_LANES;
    for (int c0 = 0; c0 < s.V; c0 += cols) {
        const int c = c0 + tid / DR_LANES;
        const bool there = c < s.V;
        const float* from = (STAGED ? held : head_state) + static_cast<size_t>(there ? c : 0) * DP;
        float* to = head_state + static_cast<size_t>(there ? c : 0) * DP;
        float S[R];
#pragma unroll
        for (int j = 0; j < R / 4; ++j) {
            const float4 x = *reinterpret_cast<const float4*>(from + 4 * l + 32 * j);
            S[4 * j] = x.x; S[4 * j + 1] = x.y; S[4 * j + 2] = x.z; S[4 * j + 3] = x.w;
        }
        const float o = dr_token<R>(S, sk, sq, sg, l, there ? sv[c] : 0.0f, beta, kq);
        if (there) {
#pragma unroll
            for (int j = 0; j < R / 4; ++j)
                *reinterpret_cast<float4*>(to + 4 * l + 32 * j) = make_float4(S[4 * j], S[4 * j + 1], S[4 * j + 2], S[4 * j + 3]);
            if (l == 0) so[c] = o;
        }
    }
    __syncthreads();
    float ss = 0.0f;
    for (int c = tid; c < s.V; c += nthreads) ss += so[c] * so[c];
    const float total = block_sum(ss, red);
    const float inv = 1.0f / sqrtf(total / static_cast<float>(s.V) + eps);
    TO* orow = out + t * out_stride + out_off + h * s.V;
    for (int c = tid; c < s.V; c += nthreads) orow[c] = from_f32<TO>(so[c] * inv * norm_w[c] * sgate[c] * out_scale);
}

// D rounded up to what the kernels are instantiated for: 32, 64, 128, 256; 0: larger.
extern "C" int llm_delta_padded(int D) { return D <= 0 ? 0 : D <= 32 ? 32 : D <= 64 ? 64 : D <= 128 ? 128 : D <= 256 ? 256 : 0; }

extern "C" int llm_delta_supported(int D, int V) { return llm_delta_padded(D) > 0 && V > 0 && V <= 1024; }

static int delta_shape(DeltaShape& s, int H, int G, int D, int V, int taps, int q_off, int b_off, int a_off, int ra, int g_off,
                       int rg, long long stride, long long slot_stride) {
    const int DP = llm_delta_padded(D);
    if (H <= 0 || G <= 0 || H % G || !llm_delta_supported(D, V) || taps < 1 || ra <= 0 || rg <= 0 || ra > 1024 || rg > 1024 || H > 65535)
        return LLM_REFUSED_SIZE;
    const long long ring_off = static_cast<long long>(H) * V * DP;
    if (slot_stride < ring_off + static_cast<long long>(taps) * (2LL * G * D + static_cast<long long>(H) * V) || slot_stride % 4)
        return LLM_REFUSED_SIZE;
    s = {H, G, D, V, DP, (V + 3) / 4 * 4, taps, q_off, q_off + G * D, q_off + 2 * G * D, b_off, a_off, ra, g_off, rg,
         stride, slot_stride, ring_off};
    return LLM_OK;
}

// Everything of a step that is not all single tokens.  Scratch (float32): qn, kn [T, G, DP], vn [T, H, VP], beta [T, H],
// decay [T, H, DP] (whose places from D on must be finite), gate and o [T, H, V], pk and pq [T, H, DP], and for P =
// T / 4 + entries + 1 chunks total [P, H, DP] and num [P, H, 24].
// `conv_w` [C, taps]: the rows of q, k and v one after another.
extern "C" int llm_delta_scan(
    const float* proj, long long stride, int q_off, int b_off, int a_off, int ra, int g_off, int rg, const float* conv_w, int taps,
    const void* wa, const void* wg, int w_dtype, const float* dt_bias, const float* a_log, const float* norm_w, float eps,
    float out_scale, void* out, int out_dtype, long long out_stride, int out_off, float* state, long long slot_stride,
    const int32_t* positions, const int32_t* token_entry, const int32_t* entry_slot, const int32_t* entry_q_start,
    const int32_t* entry_q_len, int num_tokens, int num_entries, int H, int G, int D, int V, float* qn, float* kn, float* vn,
    float* beta, float* decay, float* gate, float* o, float* pk, float* pq, float* total, float* num, uintptr_t stream) {
    if (num_tokens <= 0 || num_entries <= 0) return LLM_OK;
    DeltaShape s;
    const int rc = delta_shape(s, H, G, D, V, taps, q_off, b_off, a_off, ra, g_off, rg, stride, slot_stride);
    if (rc != LLM_OK) return rc;
    if (!aligned16(state) || !aligned16(qn) || !aligned16(kn) || !aligned16(vn) || !aligned16(decay) || !aligned16(pk) || !aligned16(pq) ||
        !aligned16(total) || !aligned16(num))
        return LLM_REFUSED_ALIGN;
    if (w_dtype != LLM_DT_F32 && w_dtype != LLM_DT_BF16) return LLM_REFUSED_DTYPE;
    if (out_dtype != LLM_DT_F32 && out_dtype != LLM_DT_BF16) return LLM_REFUSED_DTYPE;
    cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
    const dim3 pgrid((num_tokens + DP_TOKENS - 1) / DP_TOKENS, (2 * G + H + DP_WARPS - 1) / DP_WARPS);
#define PREPARE(PER)                                                                                                  \
    launch_pdl((delta_prepare_kernel<PER>), pgrid, dim3(DP_WARPS * 32), 0, st, s, proj, conv_w, state, positions,      \
               token_entry, entry_slot, entry_q_start, qn, kn, vn, beta, num_tokens)
    switch (s.DP) {
        case 32: PREPARE(1); break;
        case 64: PREPARE(2); break;
        case 128: PREPARE(4); break;
        default: PREPARE(8); break;
    }
#undef PREPARE
    const int da = (H * D + DL_CHANNELS - 1) / DL_CHANNELS, ga = (H * V + DL_CHANNELS - 1) / DL_CHANNELS;
    const dim3 lgrid((num_tokens + DL_TOKENS - 1) / DL_TOKENS, da + ga);
    const size_t lsmem = static_cast<size_t>(DL_PITCH) * (ra > rg ? ra : rg) * sizeof(float);
    if (lgrid.y > 65535) return LLM_REFUSED_SIZE;
#define LOWRANK(TW)                                                                                                   \
    do {                                                                                                              \
        auto kern = delta_lowrank_kernel<TW>;                                                                         \
        if (lsmem > 48 * 1024) {                                                                                      \
            const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize,             \
                                                       static_cast<int>(lsmem));                                      \
            if (e != cudaSuccess) return static_cast<int>(e);                                                         \
        }                                                                                                             \
        launch_pdl(kern, lgrid, dim3(DL_THREADS), lsmem, st, s, proj, static_cast<const TW*>(wa), dt_bias, a_log,    \
                   static_cast<const TW*>(wg), decay, gate, num_tokens, da);                                          \
    } while (0)
    if (w_dtype == LLM_DT_F32) LOWRANK(float);
    else LOWRANK(bf16);
#undef LOWRANK
    const dim3 cgrid(num_tokens, (H + DC_WARPS - 1) / DC_WARPS);
#define CHUNKS_OF(DP)                                                                                                 \
    launch_pdl((delta_chunk_kernel<DP>), cgrid, dim3(DC_WARPS * 32), 0, st, s, qn, kn, decay, pk, pq, total, num,      \
               token_entry, entry_q_start, entry_q_len, num_tokens)
    switch (s.DP) {
        case 32: CHUNKS_OF(32); break;
        case 64: CHUNKS_OF(64); break;
        case 128: CHUNKS_OF(128); break;
        default: CHUNKS_OF(256); break;
    }
#undef CHUNKS_OF
#define SCAN(DP, C, WARPS)                                                                                            \
    do {                                                                                                              \
        auto kern = delta_scan_kernel<DP, C, WARPS>;                                                                  \
        constexpr int K = DP >= 128 ? 1 : 128 / DP, COLS = WARPS * K * C, CH = DR_TB / DR_CHUNK;                      \
        const size_t smem = (2 * (static_cast<size_t>(DR_TB) * (3 * DP + COLS + 1) + CH * (DP + DR_NUM)) + COLS * 8) * sizeof(float); \
        if (smem > 48 * 1024) {                                                                                       \
            const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize,             \
                                                       static_cast<int>(smem));                                       \
            if (e != cudaSuccess) return static_cast<int>(e);                                                         \
        }                                                                                                             \
        launch_pdl(kern, dim3(num_entries, H, (V + COLS - 1) / COLS), dim3(WARPS * 32), smem, st, s, proj, pq, pk, vn, \
                   beta, decay, total, num, o, state, positions, entry_slot, entry_q_start, entry_q_len);             \
    } while (0)
    // few columns: fewer a warp, so that more schedulers have one; many: more a warp, which costs fewer instructions a column
    const long long columns = static_cast<long long>(num_entries) * H * V;
    const int plan = columns <= 640 ? 0 : columns <= 1300 ? 1 : columns <= 3000 ? 2 : 3;
    switch (s.DP) {
        case 32: SCAN(32, 2, 2); break;
        case 64: SCAN(64, 2, 4); break;
        case 128:
            if (plan == 0) SCAN(128, 1, 4);
            else if (plan == 1) SCAN(128, 2, 4);
            else if (plan == 2) SCAN(128, 2, 8);
            else SCAN(128, 4, 4);
            break;
        default:
            if (plan == 0) SCAN(256, 1, 4);
            else SCAN(256, 2, 4);
            break;
    }
#undef SCAN
    const long long items = static_cast<long long>(num_tokens) * H;
    const long long oblocks = (items + 3) / 4;
    if (oblocks > 0x7fffffffLL) return LLM_REFUSED_SIZE;
    if (out_dtype == LLM_DT_F32)
        launch_pdl((delta_output_kernel<float>), dim3(static_cast<unsigned>(oblocks)), dim3(128), 0, st, o, gate, norm_w, eps, out_scale,
                   static_cast<float*>(out), out_stride, out_off, H, V, items);
    else
        launch_pdl((delta_output_kernel<bf16>), dim3(static_cast<unsigned>(oblocks)), dim3(128), 0, st, o, gate, norm_w, eps, out_scale,
                   static_cast<bf16*>(out), out_stride, out_off, H, V, items);
    return launch_status();
}

// A step whose entries all bring one token.
extern "C" int llm_delta_step(
    const float* proj, long long stride, int q_off, int b_off, int a_off, int ra, int g_off, int rg, const float* conv_w, int taps,
    const void* wa, const void* wg, int w_dtype, const float* dt_bias, const float* a_log, const float* norm_w, float eps,
    float out_scale, void* out, int out_dtype, long long out_stride, int out_off, float* state, long long slot_stride,
    const int32_t* positions, const int32_t* entry_slot, const int32_t* entry_q_start, int num_entries, int H, int G, int D, int V,
    uintptr_t stream) {
    if (num_entries <= 0) return LLM_OK;
    DeltaShape s;
    const int rc = delta_shape(s, H, G, D, V, taps, q_off, b_off, a_off, ra, g_off, rg, stride, slot_stride);
    if (rc != LLM_OK) return rc;
    if (!aligned16(state)) return LLM_REFUSED_ALIGN;
    int threads = V * DR_LANES;
    // few blocks: as fast as one can be; many: small ones, three to an SM, that overlap
    const bool few = static_cast<long long>(num_entries) * H <= 2 * 148;
    const int most = few ? 512 : 256;
    threads = threads > most ? most : (threads + 31) / 32 * 32;
    if (threads < 128) threads = 128;
    int parts = threads / (D + V);
    parts = parts < 1 ? 1 : parts > 8 ? 8 : parts;
    const size_t base = (3 * static_cast<size_t>(s.DP) + 36 + 3 * V + ra + rg + static_cast<size_t>(parts) * (D + V) + 3) / 4 * 4 * sizeof(float);
    const int esz = w_dtype == LLM_DT_F32 ? 4 : 2, per = 16 / esz;
    const size_t held = static_cast<size_t>(V) * s.DP * sizeof(float), low = (static_cast<size_t>(ra) * D + static_cast<size_t>(rg) * V) * esz;
    const bool vec = D % per == 0 && V % per == 0 && aligned16(wa) && aligned16(wg);
    const bool staged = base + held <= 200 * 1024;
    const int low_staged = staged && vec && base + held + low <= 200 * 1024 && few;
    const size_t smem = base + (staged ? held : 0) + (low_staged ? low : 0);
    if (smem > 200 * 1024) return LLM_REFUSED_SIZE;
    cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
    const dim3 grid(num_entries, H);
#define STEP(R, TW, TO)                                                                                               \
    do {                                                                                                              \
        auto kern = staged ? delta_step_kernel<R, TW, TO, true> : delta_step_kernel<R, TW, TO, false>;                \
        if (smem > 48 * 1024) {                                                                                       \
            const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize,             \
                                                       static_cast<int>(smem));                                       \
            if (e != cudaSuccess) return static_cast<int>(e);                                                         \
        }                                                                                                             \
        launch_pdl(kern, grid, dim3(threads), smem, st, s, proj, conv_w, static_cast<const TW*>(wa), dt_bias, a_log,  \
                   static_cast<const TW*>(wg), norm_w, eps, out_scale, static_cast<TO*>(out), out_stride, out_off,    \
                   state, positions, entry_slot, entry_q_start, low_staged);                                          \
    } while (0)
#define BY_R(TW, TO)                                                                                                  \
    switch (s.DP) {                                                                                                   \
        case 32: STEP(4, TW, TO); break;                                                                              \
        case 64: STEP(8, TW, TO); break;                                                                              \
        case 128: STEP(16, TW, TO); break;                                                                            \
        default: STEP(32, TW, TO); break;                                                                             \
    }
    if (w_dtype == LLM_DT_F32 && out_dtype == LLM_DT_F32) { BY_R(float, float) }
    else if (w_dtype == LLM_DT_F32 && out_dtype == LLM_DT_BF16) { BY_R(float, bf16) }
    else if (w_dtype == LLM_DT_BF16 && out_dtype == LLM_DT_BF16) { BY_R(bf16, bf16) }
    else if (w_dtype == LLM_DT_BF16 && out_dtype == LLM_DT_F32) { BY_R(bf16, float) }
    else return LLM_REFUSED_DTYPE;
#undef BY_R
#undef STEP
    return launch_status();
}
