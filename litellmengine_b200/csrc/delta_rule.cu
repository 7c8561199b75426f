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
// The columns of S do not touch one another: column v needs k, q, g of the head and its own v_t.  So a column is
// eight neighbouring lanes of a warp, each holding R of its rows (rows 4 l + 32 j .. + 3 of lane l, so that the eight
// lanes read 128 contiguous bytes of k, q or g), and the only exchange per token is a sum over eight lanes.  Both
// products with the decayed state are taken before the write, o = (gS)^T q + (k . q) u, so their sums travel
// together; k . q is one number per (token, key head), made beforehand.  Blocks take any number of columns of
// any head: a long prompt of one request spreads over as many SMs as it has columns, without being cut in time.
//
//   delta_prepare_kernel   a warp per (token, key head): convolution, silu, unit norm of q and k, and k . q; a warp per
//                          (token, value head): convolution and silu of v, beta
//   delta_lowrank_kernel   the second halves of both low-rank projections: decays and gates
//   delta_scan_kernel      one block per (entry, head, columns): the recurrence over the entry's tokens, staged sixteen
//                          at a time with cp.async into two buffers; o in 32-bit; keeps the convolutions' last inputs
//   delta_output_kernel    a warp per (token, head): norm, weight, gate, scale, store in the compute dtype
//   delta_step_kernel      all of it for entries of ONE token (decode steps): the state streams through once
//
// Per request slot the mixer keeps one row of floats: S of every head transposed, [H][V][DP] (DP = D rounded up to
// 32, 64, 128 or 256; rows from D on stay zero), then a ring of `taps` rows of the C = 2 G D + H V convolved
// projections; the row of the token at position p sits at ring row p mod taps.  A token reads the rows of positions
// p - 1 .. p - taps + 1 and writes row p mod taps, which is none of those, so in a decode step blocks that share a
// key head may read the ring while one of them writes it.
#include "common.cuh"

#define DR_TB 16            // tokens staged at a time
#define DR_LANES 8          // lanes a column of the state is spread over

__device__ __forceinline__ void dr_cp16(float* smem_dst, const float* src) {
    const unsigned d = static_cast<unsigned>(__cvta_generic_to_shared(smem_dst));
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(d), "l"(src));
}

__device__ __forceinline__ float dr_silu(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float dr_sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float dr_softplus(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }
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
// grid: (tokens, ceil((G + H) / DP_WARPS)).  PER: registers a lane needs for a head's channels, ceil(DP / 32).
template <int PER>
__global__ void delta_prepare_kernel(const DeltaShape s, const float* __restrict__ proj, const float* __restrict__ conv_w,
                                     const float* __restrict__ state, const int32_t* __restrict__ positions,
                                     const int32_t* __restrict__ token_entry, const int32_t* __restrict__ entry_slot,
                                     const int32_t* __restrict__ entry_q_start, float* __restrict__ qn, float* __restrict__ kn,
                                     float* __restrict__ vn, float* __restrict__ kq, float* __restrict__ beta) {
    pdl_begin();
    const long long t = blockIdx.x;
    const int item = blockIdx.y * DP_WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (item >= s.G + s.H) return;
    const int e = token_entry[t], pos = positions[t];
    const long long row0 = entry_q_start[e];
    const float* ring = state + entry_slot[e] * s.slot_stride + s.ring_off;
    if (item < s.G) {
        const int c0 = item * s.D;
        float q[PER], k[PER], qq = 0.0f, kk = 0.0f, dot = 0.0f;
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int d = lane + 32 * i;
            q[i] = k[i] = 0.0f;
            if (d < s.D) {
                q[i] = dr_silu(dr_conv(s, proj, conv_w, ring, t, row0, pos, c0 + d));
                k[i] = dr_silu(dr_conv(s, proj, conv_w, ring, t, row0, pos, s.G * s.D + c0 + d));
            }
            qq += q[i] * q[i];
            kk += k[i] * k[i];
        }
        qq = warp_sum(qq);
        kk = warp_sum(kk);
        const float iq = 1.0f / sqrtf(qq + 1e-6f) / sqrtf(static_cast<float>(s.D)), ik = 1.0f / sqrtf(kk + 1e-6f);
        const size_t at = (static_cast<size_t>(t) * s.G + item) * s.DP;
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            q[i] *= iq;
            k[i] *= ik;
            dot += q[i] * k[i];
            qn[at + lane + 32 * i] = q[i];                     // rows from D on: zeros
            kn[at + lane + 32 * i] = k[i];
        }
        dot = warp_sum(dot);
        if (lane == 0) kq[static_cast<size_t>(t) * s.G + item] = dot;
    } else {
        const int h = item - s.G;
        float* o = vn + (static_cast<size_t>(t) * s.H + h) * s.VP;
        for (int c = lane; c < s.VP; c += 32)
            o[c] = c < s.V ? dr_silu(dr_conv(s, proj, conv_w, ring, t, row0, pos, 2 * s.G * s.D + h * s.V + c)) : 0.0f;
        if (lane == 0) beta[static_cast<size_t>(t) * s.H + h] = dr_sigmoid(proj[t * s.stride + s.b_off + h]);
    }
}

// Second halves of the low-rank projections.  A block takes DL_TOKENS tokens and DL_CHANNELS channels (one a thread) of
// either the decays or the gates; the tokens' first halves sit in shared memory as [rank][tokens], so that a thread
// reads four tokens' values at a time and each weight serves all of the block's tokens.  Weights are transposed,
// [rank][channels].
#define DL_TOKENS 32
#define DL_CHANNELS 128
template <typename TW>
__global__ void delta_lowrank_kernel(const DeltaShape s, const float* __restrict__ proj, const TW* __restrict__ wa,
                                     const float* __restrict__ dt_bias, const float* __restrict__ a_log,
                                     const TW* __restrict__ wg, float* __restrict__ decay, float* __restrict__ gate,
                                     int num_tokens, int decay_blocks) {
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
        a[j * DL_TOKENS + t] = t < nt ? proj[static_cast<size_t>(t0 + t) * s.stride + off + j] : 0.0f;
    }
    __syncthreads();
    const int c = (is_decay ? blockIdx.y : blockIdx.y - decay_blocks) * DL_CHANNELS + threadIdx.x;
    if (c >= channels) return;
    float z[DL_TOKENS];
    const float bias = is_decay ? dt_bias[c] : 0.0f;
#pragma unroll
    for (int t = 0; t < DL_TOKENS; ++t) z[t] = bias;
    for (int j0 = 0; j0 < rank; j0 += 8) {                      // eight weights in flight
        float wv[8];
#pragma unroll
        for (int u = 0; u < 8; ++u) wv[u] = j0 + u < rank ? to_f32(w[static_cast<size_t>(j0 + u) * channels + c]) : 0.0f;
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            const float4* ar = reinterpret_cast<const float4*>(a + min(j0 + u, rank - 1) * DL_TOKENS);
#pragma unroll
            for (int t = 0; t < DL_TOKENS; t += 4) {
                const float4 v = ar[t >> 2];
                z[t] += wv[u] * v.x;
                z[t + 1] += wv[u] * v.y;
                z[t + 2] += wv[u] * v.z;
                z[t + 3] += wv[u] * v.w;
            }
        }
    }
    if (is_decay) {
        const int h = c / s.D, d = c - h * s.D;
        const float ea = expf(a_log[h]);
#pragma unroll
        for (int t = 0; t < DL_TOKENS; ++t)
            if (t < nt) decay[(static_cast<size_t>(t0 + t) * s.H + h) * s.DP + d] = dr_decay(z[t], ea);
    } else {
#pragma unroll
        for (int t = 0; t < DL_TOKENS; ++t)
            if (t < nt) gate[static_cast<size_t>(t0 + t) * channels + c] = dr_sigmoid(z[t]);
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

// grid (entries, H, column tiles); COLS columns a block, COLS * 8 threads.
template <int R, int COLS>
__global__ void __launch_bounds__(COLS * DR_LANES) delta_scan_kernel(
    const DeltaShape s, const float* __restrict__ proj, const float* __restrict__ qn, const float* __restrict__ kn,
    const float* __restrict__ vn, const float* __restrict__ kq, const float* __restrict__ beta,
    const float* __restrict__ decay, float* __restrict__ o, float* __restrict__ state,
    const int32_t* __restrict__ positions, const int32_t* __restrict__ entry_slot,
    const int32_t* __restrict__ entry_q_start, const int32_t* __restrict__ entry_q_len) {
    pdl_begin();
    constexpr int DP = DR_LANES * R, THREADS = COLS * DR_LANES;
    constexpr int BUF = DR_TB * (3 * DP + COLS + 2);            // q, k, g, v, then beta and k . q of a batch of tokens
    extern __shared__ __align__(16) float smem[];
    float* part = smem + 2 * BUF;                               // [DR_TB][COLS]: the batch's outputs
    const int entry = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int kvh = h / (s.H / s.G), c0 = blockIdx.z * COLS;
    const int l = tid & (DR_LANES - 1), col = tid / DR_LANES, c = c0 + col;
    const long long row0 = entry_q_start[entry];
    const int count = entry_q_len[entry];
    float* slot = state + entry_slot[entry] * s.slot_stride;
    float* col_state = slot + (static_cast<long long>(h) * s.V + c) * DP;
    float S[R];
#pragma unroll
    for (int j = 0; j < R / 4; ++j) {
        const float4 x = c < s.V ? *reinterpret_cast<const float4*>(col_state + 4 * l + 32 * j) : make_float4(0, 0, 0, 0);
        S[4 * j] = x.x; S[4 * j + 1] = x.y; S[4 * j + 2] = x.z; S[4 * j + 3] = x.w;
    }
    auto stage = [&](int done, int buf) {
        const int nb = min(DR_TB, count - done);
        float* bq = smem + buf * BUF;
        float* bk = bq + DR_TB * DP;
        float* bg = bk + DR_TB * DP;
        float* bv = bg + DR_TB * DP;
        float* bs = bv + DR_TB * COLS;
        for (int idx = tid; idx < nb * (DP / 4); idx += THREADS) {
            const int tok = idx / (DP / 4), x = (idx - tok * (DP / 4)) * 4;
            const size_t t = static_cast<size_t>(row0 + done + tok);
            dr_cp16(bq + tok * DP + x, qn + (t * s.G + kvh) * DP + x);
            dr_cp16(bk + tok * DP + x, kn + (t * s.G + kvh) * DP + x);
            dr_cp16(bg + tok * DP + x, decay + (t * s.H + h) * DP + x);
        }
        for (int idx = tid; idx < nb * (COLS / 4); idx += THREADS) {
            const int tok = idx / (COLS / 4), x = (idx - tok * (COLS / 4)) * 4;
            if (c0 + x < s.VP)
                dr_cp16(bv + tok * COLS + x, vn + (static_cast<size_t>(row0 + done + tok) * s.H + h) * s.VP + c0 + x);
        }
        if (tid < nb) {
            const size_t t = static_cast<size_t>(row0 + done + tid);
            bs[tid] = beta[t * s.H + h];
            bs[DR_TB + tid] = kq[t * s.G + kvh];
        }
        asm volatile("cp.async.commit_group;\n" ::);
    };
    stage(0, 0);
    for (int done = 0, b = 0; done < count; done += DR_TB, ++b) {
        const int nb = min(DR_TB, count - done);
        const bool more = done + DR_TB < count;
        if (more) {
            stage(done + DR_TB, (b + 1) & 1);
            asm volatile("cp.async.wait_group 1;\n" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        }
        __syncthreads();
        const float* bq = smem + (b & 1) * BUF;
        const float* bk = bq + DR_TB * DP;
        const float* bg = bk + DR_TB * DP;
        const float* bv = bg + DR_TB * DP;
        const float* bs = bv + DR_TB * COLS;
#pragma unroll 2
        for (int tok = 0; tok < nb; ++tok) {
            const float out = dr_token<R>(S, bk + tok * DP, bq + tok * DP, bg + tok * DP, l, bv[tok * COLS + col], bs[tok],
                                          bs[DR_TB + tok]);
            if (l == 0) part[tok * COLS + col] = out;
        }
        __syncthreads();
        for (int idx = tid; idx < nb * COLS; idx += THREADS) {
            const int tok = idx / COLS, x = idx - tok * COLS;
            if (c0 + x < s.V) o[(static_cast<size_t>(row0 + done + tok) * s.H + h) * s.V + c0 + x] = part[idx];
        }
    }
    if (c < s.V) {
#pragma unroll
        for (int j = 0; j < R / 4; ++j)
            *reinterpret_cast<float4*>(col_state + 4 * l + 32 * j) = make_float4(S[4 * j], S[4 * j + 1], S[4 * j + 2], S[4 * j + 3]);
    }
    // the convolutions' inputs of the portion's last tokens (the kernel before this one has read the ring)
    const int C = 2 * s.G * s.D + s.H * s.V, keep = min(count, s.taps - 1);
    float* ring = slot + s.ring_off;
    const bool with_qk = blockIdx.z == 0 && h % (s.H / s.G) == 0;
    for (int i = 0; i < keep; ++i) {
        const long long t = row0 + count - keep + i;
        float* dst = ring + static_cast<long long>(positions[t] % s.taps) * C;
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

// Entries that bring one token: one block per (entry, head), V columns walked blockDim / 8 at a time.
template <int R, typename TW, typename TO>
__global__ void __launch_bounds__(1024) delta_step_kernel(
    const DeltaShape s, const float* __restrict__ proj, const float* __restrict__ conv_w, const TW* __restrict__ wa,
    const float* __restrict__ dt_bias, const float* __restrict__ a_log, const TW* __restrict__ wg,
    const float* __restrict__ norm_w, float eps, float out_scale, TO* __restrict__ out, long long out_stride, int out_off,
    float* __restrict__ state, const int32_t* __restrict__ positions, const int32_t* __restrict__ entry_slot,
    const int32_t* __restrict__ entry_q_start) {
    pdl_begin();
    constexpr int DP = DR_LANES * R;
    extern __shared__ __align__(16) float smem[];
    float* sq = smem;                         // [DP] each
    float* sk = sq + DP;
    float* sg = sk + DP;
    float* sv = sg + DP;                      // [V]
    float* so = sv + s.V;                     // [V]
    float* sgate = so + s.V;                  // [V]
    float* red = sgate + s.V;                 // 36
    float* first = red + 36;                  // [ra + rg]: the first halves of the low-rank projections
    float* split = first + s.ra + s.rg;       // [parts][D + V]
    const int entry = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, nthreads = blockDim.x;
    const int kvh = h / (s.H / s.G);
    const long long t = entry_q_start[entry];
    const int pos = positions[t];
    const float* pr = proj + t * s.stride;
    float* slot = state + entry_slot[entry] * s.slot_stride;
    float* ring = slot + s.ring_off;
    const int C = 2 * s.G * s.D + s.H * s.V;
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
    __syncthreads();
    // low-rank second halves: `parts` threads share a channel's sum
    const int chans = s.D + s.V;
    int parts = nthreads / chans;
    if (parts < 1) parts = 1;
    if (parts > 8) parts = 8;
    for (int i = tid; i < parts * chans; i += nthreads) {
        const int p = i / chans, ch = i - p * chans;
        const bool is_decay = ch < s.D;
        const int rank = is_decay ? s.ra : s.rg, width = is_decay ? s.H * s.D : s.H * s.V;
        const TW* w = is_decay ? wa + h * s.D + ch : wg + h * s.V + (ch - s.D);
        const float* a = is_decay ? first : first + s.ra;
        const int per = (rank + parts - 1) / parts, j1 = min(rank, (p + 1) * per);
        float z = 0.0f;
        int j = p * per;
        for (; j + 8 <= j1; j += 8) {
            float wv[8];
#pragma unroll
            for (int u = 0; u < 8; ++u) wv[u] = to_f32(w[static_cast<size_t>(j + u) * width]);
#pragma unroll
            for (int u = 0; u < 8; ++u) z += wv[u] * a[j + u];
        }
        for (; j < j1; ++j) z += to_f32(w[static_cast<size_t>(j) * width]) * a[j];
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
                g = dr_decay(z, expf(a_log[h]));
            }
            sg[i] = g;
        } else {
            float z = 0.0f;
            for (int p = 0; p < parts; ++p) z += split[p * chans + s.D + (i - DP)];
            sgate[i - DP] = dr_sigmoid(z);
        }
    }
    __syncthreads();
    const float beta = dr_sigmoid(pr[s.b_off + h]), kq = red[33];
    const int l = tid & (DR_LANES - 1), cols = nthreads / DR_LANES;
    for (int c0 = 0; c0 < s.V; c0 += cols) {
        const int c = c0 + tid / DR_LANES;
        const bool there = c < s.V;
        float* col_state = slot + (static_cast<long long>(h) * s.V + (there ? c : 0)) * DP;
        float S[R];
#pragma unroll
        for (int j = 0; j < R / 4; ++j) {
            const float4 x = *reinterpret_cast<const float4*>(col_state + 4 * l + 32 * j);
            S[4 * j] = x.x; S[4 * j + 1] = x.y; S[4 * j + 2] = x.z; S[4 * j + 3] = x.w;
        }
        const float o = dr_token<R>(S, sk, sq, sg, l, there ? sv[c] : 0.0f, beta, kq);
        if (there) {
#pragma unroll
            for (int j = 0; j < R / 4; ++j)
                *reinterpret_cast<float4*>(col_state + 4 * l + 32 * j) = make_float4(S[4 * j], S[4 * j + 1], S[4 * j + 2], S[4 * j + 3]);
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

// Everything of a step that is not all single tokens.  Scratch (float32): qn, kn [T, G, DP], vn [T, H, VP], kq [T, G],
// beta [T, H], decay [T, H, DP] (whose places from D on must be finite), gate and o [T, H, V].
// `conv_w` [C, taps]: the rows of q, k and v one after another.
extern "C" int llm_delta_scan(
    const float* proj, long long stride, int q_off, int b_off, int a_off, int ra, int g_off, int rg, const float* conv_w, int taps,
    const void* wa, const void* wg, int w_dtype, const float* dt_bias, const float* a_log, const float* norm_w, float eps,
    float out_scale, void* out, int out_dtype, long long out_stride, int out_off, float* state, long long slot_stride,
    const int32_t* positions, const int32_t* token_entry, const int32_t* entry_slot, const int32_t* entry_q_start,
    const int32_t* entry_q_len, int num_tokens, int num_entries, int H, int G, int D, int V, float* qn, float* kn, float* vn,
    float* kq, float* beta, float* decay, float* gate, float* o, uintptr_t stream) {
    if (num_tokens <= 0 || num_entries <= 0) return LLM_OK;
    DeltaShape s;
    const int rc = delta_shape(s, H, G, D, V, taps, q_off, b_off, a_off, ra, g_off, rg, stride, slot_stride);
    if (rc != LLM_OK) return rc;
    if (!aligned16(state) || !aligned16(qn) || !aligned16(kn) || !aligned16(vn) || !aligned16(decay)) return LLM_REFUSED_ALIGN;
    if (w_dtype != LLM_DT_F32 && w_dtype != LLM_DT_BF16) return LLM_REFUSED_DTYPE;
    if (out_dtype != LLM_DT_F32 && out_dtype != LLM_DT_BF16) return LLM_REFUSED_DTYPE;
    cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
    const dim3 pgrid(num_tokens, (G + H + DP_WARPS - 1) / DP_WARPS);
#define PREPARE(PER)                                                                                                  \
    launch_pdl((delta_prepare_kernel<PER>), pgrid, dim3(DP_WARPS * 32), 0, st, s, proj, conv_w, state, positions,      \
               token_entry, entry_slot, entry_q_start, qn, kn, vn, kq, beta)
    switch (s.DP) {
        case 32: PREPARE(1); break;
        case 64: PREPARE(2); break;
        case 128: PREPARE(4); break;
        default: PREPARE(8); break;
    }
#undef PREPARE
    const int da = (H * D + DL_CHANNELS - 1) / DL_CHANNELS, ga = (H * V + DL_CHANNELS - 1) / DL_CHANNELS;
    const dim3 lgrid((num_tokens + DL_TOKENS - 1) / DL_TOKENS, da + ga);
    const size_t lsmem = static_cast<size_t>(DL_TOKENS) * (ra > rg ? ra : rg) * sizeof(float);
    if (lgrid.y > 65535) return LLM_REFUSED_SIZE;
#define LOWRANK(TW)                                                                                                   \
    do {                                                                                                              \
        auto kern = delta_lowrank_kernel<TW>;                                                                         \
        if (lsmem > 48 * 1024) {                                                                                      \
            const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize,             \
                                                       static_cast<int>(lsmem));                                      \
            if (e != cudaSuccess) return static_cast<int>(e);                                                         \
        }                                                                                                             \
        launch_pdl(kern, lgrid, dim3(DL_CHANNELS), lsmem, st, s, proj, static_cast<const TW*>(wa), dt_bias, a_log,    \
                   static_cast<const TW*>(wg), decay, gate, num_tokens, da);                                          \
    } while (0)
    if (w_dtype == LLM_DT_F32) LOWRANK(float);
    else LOWRANK(bf16);
#undef LOWRANK
#define SCAN(R, COLS)                                                                                                 \
    do {                                                                                                              \
        auto kern = delta_scan_kernel<R, COLS>;                                                                       \
        const size_t smem = (2 * static_cast<size_t>(DR_TB) * (3 * DR_LANES * R + COLS + 2) + DR_TB * COLS) * sizeof(float); \
        if (smem > 48 * 1024) {                                                                                       \
            const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize,             \
                                                       static_cast<int>(smem));                                       \
            if (e != cudaSuccess) return static_cast<int>(e);                                                         \
        }                                                                                                             \
        launch_pdl(kern, dim3(num_entries, H, (V + COLS - 1) / COLS), dim3(COLS * DR_LANES), smem, st, s, proj, qn, kn, \
                   vn, kq, beta, decay, o, state, positions, entry_slot, entry_q_start, entry_q_len);                 \
    } while (0)
    switch (s.DP) {
        case 32: SCAN(4, 16); break;
        case 64: SCAN(8, 16); break;
        case 128: SCAN(16, 16); break;
        default: SCAN(32, 16); break;
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
    threads = threads > 1024 ? 1024 : (threads + 31) / 32 * 32;
    if (threads < 128) threads = 128;
    const size_t smem = (3 * static_cast<size_t>(s.DP) + 3 * V + 36 + ra + rg + 8 * static_cast<size_t>(D + V)) * sizeof(float);
    if (smem > 200 * 1024) return LLM_REFUSED_SIZE;
    cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
    const dim3 grid(num_entries, H);
#define STEP(R, TW, TO)                                                                                               \
    do {                                                                                                              \
        auto kern = delta_step_kernel<R, TW, TO>;                                                                     \
        if (smem > 48 * 1024) {                                                                                       \
            const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize,             \
                                                       static_cast<int>(smem));                                       \
            if (e != cudaSuccess) return static_cast<int>(e);                                                         \
        }                                                                                                             \
        launch_pdl(kern, grid, dim3(threads), smem, st, s, proj, conv_w, static_cast<const TW*>(wa), dt_bias, a_log,  \
                   static_cast<const TW*>(wg), norm_w, eps, out_scale, static_cast<TO*>(out), out_stride, out_off,    \
                   state, positions, entry_slot, entry_q_start);                                                      \
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
