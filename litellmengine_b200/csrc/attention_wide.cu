// Paged causal attention on the tensor cores for keys and values whose widths are their own: bfloat16, key width dk and
// value width dv any multiples of 8 up to 256 (padded with zeros to multiples of 16 in shared memory only), keys [pages,
// nkv, page, dk] and values [pages, nkv, page, dv] with their own page strides (the halves of one tensor are the special
// case).  Ordinary softmax over the keys from `first_visible(p, window)` to p: all, a sliding window, or the query's own
// chunk.  Scores, softmax state and accumulators are 32-bit; the weights go to the second product as bfloat16.
//
//   wide_prefill_kernel   prompt portions: a CTA takes 128 query rows of one head (a warp 16) and walks tiles of 64 keys,
//                         two in shared memory.
//   wide_decode_kernel    single tokens, split over the keys: a CTA takes one token, one kv head and one of the splits;
//                         the group's query heads are the 16 rows of its products, its 4 warps take 16 keys each of
//                         every tile, two tiles in shared memory (so that two CTAs or more share an SM: a warp's
//                         work on its 16 keys is a chain of latencies).  Partial results are merged by
//                         wide_combine_kernel (maxima in the base-2 domain).
// The formulas are those of the kernels for head sizes 64 and 128 (`attention_prefill.cu`, `attention_decode.cu`); what
// differs is that rows of dk and dv entries lie in shared memory at a stride of one chunk more than they are long (an
// odd number of sixteen-byte chunks, so that eight rows fall into different banks) and that value rows are padded with
// zeros to a compile-time width DV, so that the products with them have no conditions in them.
#include "mma_tiles.cuh"
#include <math_constants.h>

#define WP_WARPS 8
#define WP_BM (16 * WP_WARPS)
#define WP_BN 64
#define WP_THREADS (32 * WP_WARPS)
#define WD_BN 64
#define WD_THREADS 128

static __host__ __device__ __forceinline__ int wide_pad(int d) { return (d + 15) / 16 * 16; }        // entries computed
static __host__ __device__ __forceinline__ int wide_row(int d) { return wide_pad(d) + 8; }           // entries from row to row
static int wide_dv(int dv) { return dv <= 64 ? 64 : dv <= 96 ? 96 : dv <= 128 ? 128 : dv <= 160 ? 160 : dv <= 192 ? 192 : 256; }

// Where a key's row and a value's row lie, found once per key.
struct WideCache {
    const bf16* keys;
    const bf16* values;
    long long key_page, value_page;      // page strides in elements
    int dk, dv, page_size, num_pages;
};

template <int DV>
__global__ void __launch_bounds__(WP_THREADS, DV <= 96 ? 2 : 1) wide_prefill_kernel(
    const bf16* __restrict__ q, bf16* __restrict__ out, const WideCache c, const int32_t* __restrict__ tiles,
    const int32_t* __restrict__ entry_slot, const int32_t* __restrict__ entry_q_start,
    const int32_t* __restrict__ entry_q_len, const int32_t* __restrict__ entry_kv_len,
    const int32_t* __restrict__ block_table, int table_stride, int nq, int nkv, int window, float scale_log2e,
    int32_t* __restrict__ status, float out_scale, long long out_stride, int out_off) {
    pdl_begin();
    extern __shared__ __align__(128) unsigned char smem_raw[];
    constexpr int ldv = DV + 8;
    const int dk16 = wide_pad(c.dk), ldk = wide_row(c.dk);
    bf16* q_s = reinterpret_cast<bf16*>(smem_raw);                    // [BM][ldk]
    bf16* k_s = q_s + WP_BM * ldk;                                    // [2][64][ldk]
    bf16* v_s = k_s + 2 * WP_BN * ldk;                                // [2][64][ldv]

    const int tile = blockIdx.y, h = blockIdx.x;
    const int kvh = h / (nq / nkv);
    const int e = tiles[2 * tile], q0 = tiles[2 * tile + 1];
    if (e < 0) return;                                                // a padding entry of the tile list: no work
    const int q_len = entry_q_len[e], past = entry_kv_len[e] - q_len;
    const int row_base = entry_q_start[e] + q0, rows_here = min(WP_BM, q_len - q0);
    const int32_t* table = block_table + static_cast<size_t>(entry_slot[e]) * table_stride;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int pos_first = past + q0, pos_last = pos_first + rows_here - 1;
    const int k_first = first_visible(pos_first, window), lo_last = first_visible(pos_last, window);
    const int k_lo = k_first / WP_BN * WP_BN;
    const int n_tiles = (pos_last - k_lo) / WP_BN + 1;

    constexpr int TPR = WP_THREADS / WP_BN;                           // threads that copy one key
    const int ld_row = tid / TPR, ld_sub = tid % TPR;
    auto load_kv = [&](int kt, int buf) {
        const int key = kt + ld_row;
        bool valid = key <= pos_last && key >= k_first;
        const bf16 *ks = c.keys, *vs = c.values;
        if (valid) {
            const int logical = key / c.page_size;
            const int page = logical < table_stride ? table[logical] : -1;
            if (page < 0 || page >= c.num_pages) {
                if (atomicCAS(status, 0, 4) == 0) status[1] = row_base;
                valid = false;
            } else {
                const long long in_page = static_cast<long long>(kvh) * c.page_size + (key - logical * c.page_size);
                ks += page * c.key_page + in_page * c.dk;
                vs += page * c.value_page + in_page * c.dv;
            }
        }
        bf16* kd = k_s + (buf * WP_BN + ld_row) * ldk;
        bf16* vd = v_s + (buf * WP_BN + ld_row) * ldv;
        for (int ch = ld_sub * 8; ch < dk16; ch += TPR * 8) cp_async16(kd + ch, ch < c.dk ? ks + ch : ks, valid && ch < c.dk);
        for (int ch = ld_sub * 8; ch < DV; ch += TPR * 8) cp_async16(vd + ch, ch < c.dv ? vs + ch : vs, valid && ch < c.dv);
    };
    {
        constexpr int TPQ = WP_THREADS / WP_BM;
        const int qr = tid / TPQ, qsub = tid % TPQ;
        const bool valid = qr < rows_here;
        const bf16* src = q + (static_cast<size_t>(row_base + (valid ? qr : 0)) * nq + h) * c.dk;
        for (int ch = qsub * 8; ch < dk16; ch += TPQ * 8) cp_async16(q_s + qr * ldk + ch, ch < c.dk ? src + ch : src, valid && ch < c.dk);
    }
    load_kv(k_lo, 0);
    cp_async_commit();

    float o[DV / 8][4];
#pragma unroll
    for (int nb = 0; nb < DV / 8; ++nb) o[nb][0] = o[nb][1] = o[nb][2] = o[nb][3] = 0.0f;
    float m0 = -CUDART_INF_F, m1 = -CUDART_INF_F, l0 = 0.0f, l1 = 0.0f;      // rows lane/4 and lane/4 + 8
    const int r0 = warp * 16 + (lane >> 2);
    const int pos0 = pos_first + r0, pos1 = pos0 + 8;
    const int lo0 = first_visible(pos0, window), lo1 = first_visible(pos1, window);
    const int warp_lo = first_visible(pos_first + warp * 16, window);         // nothing below it is any of the warp's rows' to see

    for (int it = 0; it < n_tiles; ++it) {
        const int kt = k_lo + it * WP_BN, buf = it & 1;
        cp_async_wait_all();
        __syncthreads();
        if (it + 1 < n_tiles) load_kv(kt + WP_BN, buf ^ 1);
        cp_async_commit();
        if (kt > pos_first + warp * 16 + 15 || kt + WP_BN <= warp_lo) continue;      // every key lies after, or before, what this warp's rows see
        const bf16* kd = k_s + buf * WP_BN * ldk;
        const bf16* vd = v_s + buf * WP_BN * ldv;

        float s[WP_BN / 8][4];
#pragma unroll
        for (int nb = 0; nb < WP_BN / 8; ++nb) s[nb][0] = s[nb][1] = s[nb][2] = s[nb][3] = 0.0f;
        const bf16* qa = q_s + (warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ldk + (lane >> 4) * 8;
        const bf16* ka = kd + ((lane & 7) + (lane >> 4) * 8) * ldk + ((lane >> 3) & 1) * 8;
#pragma unroll 2
        for (int kb = 0; kb < dk16; kb += 16) {
            unsigned qf[4], kf[WP_BN / 16][4];
            ldmatrix_x4(qf, qa + kb);
#pragma unroll
            for (int np = 0; np < WP_BN / 16; ++np) ldmatrix_x4(kf[np], ka + np * 16 * ldk + kb);
#pragma unroll
            for (int np = 0; np < WP_BN / 16; ++np) {
                mma_bf16(s[2 * np], qf, kf[np][0], kf[np][1]);
                mma_bf16(s[2 * np + 1], qf, kf[np][2], kf[np][3]);
            }
        }
        const bool need_mask = kt + WP_BN - 1 > pos_first || kt < lo_last;
        float mx0 = -CUDART_INF_F, mx1 = -CUDART_INF_F;
#pragma unroll
        for (int nb = 0; nb < WP_BN / 8; ++nb)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int key = kt + nb * 8 + (lane & 3) * 2 + u;
                float a = s[nb][u] * scale_log2e, b = s[nb][2 + u] * scale_log2e;
                if (need_mask) {
                    if (key > pos0 || key < lo0) a = -CUDART_INF_F;
                    if (key > pos1 || key < lo1) b = -CUDART_INF_F;
                }
                s[nb][u] = a;
                s[nb][2 + u] = b;
                mx0 = fmaxf(mx0, a);
                mx1 = fmaxf(mx1, b);
            }
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
        const float mn0 = fmaxf(m0, mx0), mn1 = fmaxf(m1, mx1);
        const float al0 = (m0 == -CUDART_INF_F) ? 0.0f : exp2f(m0 - mn0);
        const float al1 = (m1 == -CUDART_INF_F) ? 0.0f : exp2f(m1 - mn1);
        const float sub0 = (mn0 == -CUDART_INF_F) ? 0.0f : mn0, sub1 = (mn1 == -CUDART_INF_F) ? 0.0f : mn1;
        float sum0 = 0.0f, sum1 = 0.0f;
        unsigned pf[WP_BN / 16][4];
#pragma unroll
        for (int nb = 0; nb < WP_BN / 8; ++nb) {
            const float p00 = exp2f(s[nb][0] - sub0), p01 = exp2f(s[nb][1] - sub0);
            const float p10 = exp2f(s[nb][2] - sub1), p11 = exp2f(s[nb][3] - sub1);
            sum0 += p00 + p01;
            sum1 += p10 + p11;
            pf[nb >> 1][(nb & 1) * 2] = pack_bf16(p00, p01);
            pf[nb >> 1][(nb & 1) * 2 + 1] = pack_bf16(p10, p11);
        }
        sum0 += __shfl_xor_sync(0xffffffffu, sum0, 1);
        sum0 += __shfl_xor_sync(0xffffffffu, sum0, 2);
        sum1 += __shfl_xor_sync(0xffffffffu, sum1, 1);
        sum1 += __shfl_xor_sync(0xffffffffu, sum1, 2);
        l0 = l0 * al0 + sum0;
        l1 = l1 * al1 + sum1;
        m0 = mn0;
        m1 = mn1;
        const bf16* va = vd + ((lane & 7) + ((lane >> 3) & 1) * 8) * ldv + (lane >> 4) * 8;
#pragma unroll
        for (int np = 0; np < DV / 16; ++np) {
            o[2 * np][0] *= al0; o[2 * np][1] *= al0; o[2 * np][2] *= al1; o[2 * np][3] *= al1;
            o[2 * np + 1][0] *= al0; o[2 * np + 1][1] *= al0; o[2 * np + 1][2] *= al1; o[2 * np + 1][3] *= al1;
            unsigned vf[WP_BN / 16][4];
#pragma unroll
            for (int kb = 0; kb < WP_BN / 16; ++kb) ldmatrix_x4_trans(vf[kb], va + kb * 16 * ldv + np * 16);
#pragma unroll
            for (int kb = 0; kb < WP_BN / 16; ++kb) {
                mma_bf16(o[2 * np], pf[kb], vf[kb][0], vf[kb][1]);
                mma_bf16(o[2 * np + 1], pf[kb], vf[kb][2], vf[kb][3]);
            }
        }
    }
    cp_async_wait_all();

    const bool live0 = r0 < rows_here, live1 = r0 + 8 < rows_here;
    const float inv0 = live0 && l0 > 0.0f ? out_scale / l0 : 0.0f, inv1 = live1 && l1 > 0.0f ? out_scale / l1 : 0.0f;
    bf16* orow0 = out + static_cast<size_t>(row_base + r0) * out_stride + out_off + static_cast<size_t>(h) * c.dv;
    bf16* orow1 = orow0 + static_cast<size_t>(8) * out_stride;
#pragma unroll
    for (int nb = 0; nb < DV / 8; ++nb) {
        const int col = nb * 8 + (lane & 3) * 2;                     // dv is a multiple of 8: a block is in or out as a whole
        if (col >= c.dv) break;
        if (live0) *reinterpret_cast<unsigned*>(orow0 + col) = pack_bf16(o[nb][0] * inv0, o[nb][1] * inv0);
        if (live1) *reinterpret_cast<unsigned*>(orow1 + col) = pack_bf16(o[nb][2] * inv1, o[nb][3] * inv1);
    }
}

template <int DV>
__global__ void __launch_bounds__(WD_THREADS) wide_decode_kernel(
    const bf16* __restrict__ q, const WideCache c, const int32_t* __restrict__ rows, const int32_t* __restrict__ positions,
    const int32_t* __restrict__ token_entry, const int32_t* __restrict__ entry_slot,
    const int32_t* __restrict__ block_table, int table_stride, float* __restrict__ part_acc, float* __restrict__ part_ml,
    bf16* __restrict__ out, int nq, int nkv, int window, float scale_log2e, int num_splits, int32_t* __restrict__ status,
    float out_scale, long long out_stride, int out_off) {
    pdl_begin();
    extern __shared__ __align__(128) unsigned char smem_raw[];
    constexpr int ldv = DV + 8;
    const int dk16 = wide_pad(c.dk), ldk = wide_row(c.dk);
    bf16* q_s = reinterpret_cast<bf16*>(smem_raw);                 // [16][ldk]
    bf16* k_s = q_s + 16 * ldk;                                    // [2][64][ldk]
    bf16* v_s = k_s + 2 * WD_BN * ldk;                             // [2][64][ldv]
    __shared__ float m_s[4][16], l_s[4][16];

    const int split = blockIdx.x, kvh = blockIdx.y, r = blockIdx.z;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int G = nq / nkv, h0 = kvh * G;
    const int t = rows ? rows[r] : r;
    if (t < 0) return;                                              // a padding entry of the row list: no work
    const int pos = positions[t];
    const int32_t* table = block_table + static_cast<size_t>(entry_slot[token_entry[t]]) * table_stride;
    const int lo = first_visible(pos, window);
    int per_split = (pos - lo + num_splits) / num_splits;
    per_split = (per_split + WD_BN - 1) / WD_BN * WD_BN;
    const int k_begin = lo + split * per_split, k_end = min(pos + 1, k_begin + per_split);
    const int n_tiles = k_end > k_begin ? (k_end - k_begin + WD_BN - 1) / WD_BN : 0;
    const int ld_row = tid >> 1, ld_half = tid & 1;                // a pair of threads copies one key

    // the page of this thread's key is looked up one tile ahead of the copy that needs it
    auto lookup = [&](int kt) -> int {
        const int key = kt + ld_row;
        if (key >= k_end) return -2;                                // past the split: zero-fill
        const int logical = key / c.page_size;
        return logical < table_stride ? __ldg(table + logical) : -1;
    };
    auto load_kv = [&](int kt, int buf, int page) {
        const int key = kt + ld_row;
        bool valid = page >= 0;
        const bf16 *ks = c.keys, *vs = c.values;
        if (page == -1 || page >= c.num_pages) {
            if (atomicCAS(status, 0, 4) == 0) status[1] = t;
            valid = false;
        } else if (valid) {
            const long long in_page = static_cast<long long>(kvh) * c.page_size + key % c.page_size;
            ks += page * c.key_page + in_page * c.dk;
            vs += page * c.value_page + in_page * c.dv;
        }
        bf16* kd = k_s + (buf * WD_BN + ld_row) * ldk;
        bf16* vd = v_s + (buf * WD_BN + ld_row) * ldv;
#pragma unroll 4
        for (int ch = ld_half * 8; ch < dk16; ch += 16) cp_async16(kd + ch, ch < c.dk ? ks + ch : ks, valid && ch < c.dk);
#pragma unroll 4
        for (int ch = ld_half * 8; ch < DV; ch += 16) cp_async16(vd + ch, ch < c.dv ? vs + ch : vs, valid && ch < c.dv);
    };

    if (n_tiles > 0) {
        if (ld_row < 16) {                                          // the group's query heads, zero rows after them
            const bool valid = ld_row < G;
            const bf16* src = q + (static_cast<size_t>(t) * nq + h0 + (valid ? ld_row : 0)) * c.dk;
            for (int ch = ld_half * 8; ch < dk16; ch += 16) cp_async16(q_s + ld_row * ldk + ch, ch < c.dk ? src + ch : src, valid && ch < c.dk);
        }
        load_kv(k_begin, 0, lookup(k_begin));
    }
    cp_async_commit();
    int page_ahead = n_tiles > 1 ? lookup(k_begin + WD_BN) : -2;

    float o[DV / 8][4];
#pragma unroll
    for (int nb = 0; nb < DV / 8; ++nb) o[nb][0] = o[nb][1] = o[nb][2] = o[nb][3] = 0.0f;
    float m0 = -CUDART_INF_F, m1 = -CUDART_INF_F, l0 = 0.0f, l1 = 0.0f;   // rows lane/4 and lane/4 + 8
    const bf16* qa = q_s + ((lane & 7) + ((lane >> 3) & 1) * 8) * ldk + (lane >> 4) * 8;

    for (int it = 0; it < n_tiles; ++it) {
        const int kt = k_begin + it * WD_BN, buf = it & 1;
        cp_async_wait_all();
        __syncthreads();                                            // tile `it` has landed, and every warp is done with tile it-1's buffer
        if (it + 1 < n_tiles) load_kv(kt + WD_BN, buf ^ 1, page_ahead);
        cp_async_commit();
        page_ahead = it + 2 < n_tiles ? lookup(kt + 2 * WD_BN) : -2;
        const int key0 = kt + warp * 16;                            // this warp's 16 keys of the tile
        if (key0 >= k_end) continue;                                // warp-uniform: nothing of ours in this tile
        const bf16* ka = k_s + (buf * WD_BN + warp * 16 + (lane & 7) + (lane >> 4) * 8) * ldk + ((lane >> 3) & 1) * 8;
        float s[2][4], s2[2][4];                                    // even and odd blocks of 16 key entries: two chains
#pragma unroll
        for (int u = 0; u < 4; ++u) s[0][u] = s[1][u] = s2[0][u] = s2[1][u] = 0.0f;
#pragma unroll 2
        for (int kb = 0; kb < dk16; kb += 32) {
            unsigned qf[4], b[4];
            ldmatrix_x4(qf, qa + kb);
            ldmatrix_x4(b, ka + kb);
            mma_bf16(s[0], qf, b[0], b[1]);
            mma_bf16(s[1], qf, b[2], b[3]);
            if (kb + 16 < dk16) {
                unsigned qf2[4], b2[4];
                ldmatrix_x4(qf2, qa + kb + 16);
                ldmatrix_x4(b2, ka + kb + 16);
                mma_bf16(s2[0], qf2, b2[0], b2[1]);
                mma_bf16(s2[1], qf2, b2[2], b2[3]);
            }
        }
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            s[0][u] += s2[0][u];
            s[1][u] += s2[1][u];
        }
        float mx0 = -CUDART_INF_F, mx1 = -CUDART_INF_F;
#pragma unroll
        for (int nb = 0; nb < 2; ++nb)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const bool vis = key0 + nb * 8 + (lane & 3) * 2 + u < k_end;
                s[nb][u] = vis ? s[nb][u] * scale_log2e : -CUDART_INF_F;
                s[nb][2 + u] = vis ? s[nb][2 + u] * scale_log2e : -CUDART_INF_F;
                mx0 = fmaxf(mx0, s[nb][u]);
                mx1 = fmaxf(mx1, s[nb][2 + u]);
            }
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
        const float mn0 = fmaxf(m0, mx0), mn1 = fmaxf(m1, mx1);     // finite: key0 < k_end, so one key is visible
        const float al0 = (m0 == -CUDART_INF_F) ? 0.0f : exp2f(m0 - mn0);
        const float al1 = (m1 == -CUDART_INF_F) ? 0.0f : exp2f(m1 - mn1);
        const float p00 = exp2f(s[0][0] - mn0), p01 = exp2f(s[0][1] - mn0), p02 = exp2f(s[1][0] - mn0), p03 = exp2f(s[1][1] - mn0);
        const float p10 = exp2f(s[0][2] - mn1), p11 = exp2f(s[0][3] - mn1), p12 = exp2f(s[1][2] - mn1), p13 = exp2f(s[1][3] - mn1);
        float sum0 = p00 + p01 + p02 + p03, sum1 = p10 + p11 + p12 + p13;
        sum0 += __shfl_xor_sync(0xffffffffu, sum0, 1);
        sum0 += __shfl_xor_sync(0xffffffffu, sum0, 2);
        sum1 += __shfl_xor_sync(0xffffffffu, sum1, 1);
        sum1 += __shfl_xor_sync(0xffffffffu, sum1, 2);
        l0 = l0 * al0 + sum0;
        l1 = l1 * al1 + sum1;
        m0 = mn0;
        m1 = mn1;
        const unsigned pf[4] = {pack_bf16(p00, p01), pack_bf16(p10, p11), pack_bf16(p02, p03), pack_bf16(p12, p13)};
        const bf16* va = v_s + (buf * WD_BN + warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ldv + (lane >> 4) * 8;
#pragma unroll
        for (int np = 0; np < DV / 16; ++np) {
            unsigned b[4];
            ldmatrix_x4_trans(b, va + np * 16);
            o[2 * np][0] *= al0; o[2 * np][1] *= al0; o[2 * np][2] *= al1; o[2 * np][3] *= al1;
            o[2 * np + 1][0] *= al0; o[2 * np + 1][1] *= al0; o[2 * np + 1][2] *= al1; o[2 * np + 1][3] *= al1;
            mma_bf16(o[2 * np], pf, b[0], b[1]);
            mma_bf16(o[2 * np + 1], pf, b[2], b[3]);
        }
    }
    cp_async_wait_all();
    __syncthreads();                                                // tiles are done: reuse their memory

    constexpr int as = DV + 8;                                      // row stride: rows 0..3 hit different banks
    float* acc_s = reinterpret_cast<float*>(k_s);                   // [4 warps][16 rows][as]; only rows < G are used
    {
        const int r0 = lane >> 2;
        float* a0 = acc_s + (warp * 16 + r0) * as + (lane & 3) * 2;
        float* a1 = a0 + 8 * as;
#pragma unroll
        for (int nb = 0; nb < DV / 8; ++nb) {
            if (r0 < G) *reinterpret_cast<float2*>(a0 + nb * 8) = make_float2(o[nb][0], o[nb][1]);
            if (r0 + 8 < G) *reinterpret_cast<float2*>(a1 + nb * 8) = make_float2(o[nb][2], o[nb][3]);
        }
        if ((lane & 3) == 0) {
            m_s[warp][r0] = m0; l_s[warp][r0] = l0;
            m_s[warp][r0 + 8] = m1; l_s[warp][r0 + 8] = l1;
        }
    }
    __syncthreads();
    for (int i = tid; i < G * c.dv; i += WD_THREADS) {
        const int g = i / c.dv, dim = i - g * c.dv;
        const float M = fmaxf(fmaxf(m_s[0][g], m_s[1][g]), fmaxf(m_s[2][g], m_s[3][g]));
        float a = 0.0f, L = 0.0f;
#pragma unroll
        for (int w = 0; w < 4; ++w) {
            const float f = (m_s[w][g] == -CUDART_INF_F) ? 0.0f : exp2f(m_s[w][g] - M);
            if (f > 0.0f) a += acc_s[(w * 16 + g) * as + dim] * f;
            L += l_s[w][g] * f;
        }
        if (num_splits == 1) {
            out[static_cast<size_t>(t) * out_stride + out_off + (h0 + g) * c.dv + dim] = __float2bfloat16_rn(a / L * out_scale);
        } else {
            const size_t part = (static_cast<size_t>(r) * nq + h0 + g) * num_splits + split;
            part_acc[part * c.dv + dim] = a;
            if (dim == 0) {
                part_ml[part * 2] = M;
                part_ml[part * 2 + 1] = L;
            }
        }
    }
}

// One block per (token row, query head): merge the splits.
__global__ void wide_combine_kernel(const float* __restrict__ part_acc, const float* __restrict__ part_ml,
                                    const int32_t* __restrict__ rows, bf16* __restrict__ out, int nq, int dv, int num_splits,
                                    float out_scale, long long out_stride, int out_off) {
    pdl_begin();
    const int r = blockIdx.x, h = blockIdx.y;
    const int t = rows ? rows[r] : r;
    if (t < 0) return;
    const size_t first = (static_cast<size_t>(r) * nq + h) * num_splits;
    float M = -CUDART_INF_F;
    for (int s = 0; s < num_splits; ++s)
        if (part_ml[(first + s) * 2 + 1] > 0.0f) M = fmaxf(M, part_ml[(first + s) * 2]);
    for (int dim = threadIdx.x; dim < dv; dim += blockDim.x) {
        float a = 0.0f, L = 0.0f;
        for (int s = 0; s < num_splits; ++s) {
            const float ls = part_ml[(first + s) * 2 + 1];
            if (ls > 0.0f) {                          // an empty split holds nothing to add
                const float f = exp2f(part_ml[(first + s) * 2] - M);
                a += part_acc[(first + s) * dv + dim] * f;
                L += ls * f;
            }
        }
        out[static_cast<size_t>(t) * out_stride + out_off + h * dv + dim] = __float2bfloat16_rn(a / L * out_scale);
    }
}

extern "C" int llm_wide_attention_supported(int dk, int dv, int group) {
    return dk >= 8 && dk <= 256 && dk % 8 == 0 && dv >= 8 && dv <= 256 && dv % 8 == 0 && group >= 1 && group <= 16;
}

extern "C" int llm_wide_prefill_tile_rows() { return WP_BM; }

static int wide_check(const void* q, const void* keys, const void* values, long long key_page, long long value_page, int nq, int nkv,
                      int dk, int dv, int page_size) {
    if (nq <= 0 || nkv <= 0 || nq % nkv || page_size <= 0 || !llm_wide_attention_supported(dk, dv, nq / nkv)) return LLM_REFUSED_SIZE;
    if (!aligned16(q) || !aligned16(keys) || !aligned16(values) || key_page % 8 || value_page % 8) return LLM_REFUSED_ALIGN;
    return LLM_OK;
}

#define WIDE_BY_DV(LAUNCH)       \
    switch (wide_dv(dv)) {       \
        case 64: LAUNCH(64); break;   \
        case 96: LAUNCH(96); break;   \
        case 128: LAUNCH(128); break; \
        case 160: LAUNCH(160); break; \
        case 192: LAUNCH(192); break; \
        default: LAUNCH(256);    \
    }

// q: bfloat16 [T, nq*dk]; keys / values: bfloat16 [pages, nkv, page_size, dk / dv], `key_page` / `value_page` elements from
// page to page; tiles: int32 [n_tiles][2] = (entry, first query row of the tile inside the entry), each tile
// llm_wide_prefill_tile_rows() rows; the result times out_scale goes to columns out_off .. of rows of `out`, out_stride
// elements apart.  `window`: as in `first_visible`.
extern "C" int llm_wide_attention_prefill(
    const void* q, void* out, const void* keys, const void* values, long long key_page, long long value_page,
    const int32_t* tiles, int n_tiles, const int32_t* entry_slot, const int32_t* entry_q_start, const int32_t* entry_q_len,
    const int32_t* entry_kv_len, const int32_t* block_table, int table_stride, int nq, int nkv, int dk, int dv, int page_size,
    int window, float scale, int num_pages, int32_t* status, float out_scale, long long out_stride, int out_off,
    uintptr_t stream) {
    if (n_tiles <= 0) return LLM_OK;
    const int rc = wide_check(q, keys, values, key_page, value_page, nq, nkv, dk, dv, page_size);
    if (rc != LLM_OK) return rc;
    if (n_tiles > 65535) return LLM_REFUSED_SIZE;
    if (out_stride % 2 || out_off % 2 || (reinterpret_cast<uintptr_t>(out) & 3u)) return LLM_REFUSED_ALIGN;
    const size_t smem = (static_cast<size_t>(WP_BM + 2 * WP_BN) * wide_row(dk) + 2 * WP_BN * static_cast<size_t>(wide_dv(dv) + 8)) * sizeof(bf16);
    const WideCache c = {static_cast<const bf16*>(keys), static_cast<const bf16*>(values), key_page, value_page, dk, dv, page_size, num_pages};
    cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
#define LAUNCH(DD)                                                                                                         \
    do {                                                                                                                      \
        auto kern = wide_prefill_kernel<DD>;                                                                               \
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)); \
        if (e != cudaSuccess) return static_cast<int>(e);                                                                  \
        launch_pdl(kern, dim3(nq, n_tiles), dim3(WP_THREADS), smem, s, static_cast<const bf16*>(q), static_cast<bf16*>(out), c, \
                   tiles, entry_slot, entry_q_start, entry_q_len, entry_kv_len, block_table, table_stride, nq, nkv, window, \
                   scale * 1.4426950408889634f, status, out_scale, out_stride, out_off);                                   \
    } while (0)
    WIDE_BY_DV(LAUNCH)
#undef LAUNCH
    return launch_status();
}

// Floats of scratch the decode call needs: accumulators, then (maximum, sum) pairs.
extern "C" long long llm_wide_decode_scratch_floats(int n_rows, int nq, int dv, int num_splits) {
    return num_splits <= 1 ? 0 : static_cast<long long>(n_rows) * nq * num_splits * (dv + 2);
}

// The same operands; rows: int32 [n_rows] token rows to attend for (null: rows 0..n_rows-1; -1 entries are padding);
// scratch: float32, llm_wide_decode_scratch_floats long.
extern "C" int llm_wide_attention_decode(
    const void* q, void* out, const void* keys, const void* values, long long key_page, long long value_page,
    const int32_t* rows, int n_rows, const int32_t* positions, const int32_t* token_entry, const int32_t* entry_slot,
    const int32_t* block_table, int table_stride, int nq, int nkv, int dk, int dv, int page_size, int window, float scale,
    int num_pages, int num_splits, float* scratch, int32_t* status, float out_scale, long long out_stride, int out_off,
    uintptr_t stream) {
    if (n_rows <= 0) return LLM_OK;
    const int rc = wide_check(q, keys, values, key_page, value_page, nq, nkv, dk, dv, page_size);
    if (rc != LLM_OK) return rc;
    if (num_splits < 1 || num_splits > 65535 || nkv > 65535 || n_rows > 65535 || (num_splits > 1 && !scratch)) return LLM_REFUSED_SIZE;
    const size_t smem = (static_cast<size_t>(16 + 2 * WD_BN) * wide_row(dk) + static_cast<size_t>(2 * WD_BN) * (wide_dv(dv) + 8)) * sizeof(bf16);
    const WideCache c = {static_cast<const bf16*>(keys), static_cast<const bf16*>(values), key_page, value_page, dk, dv, page_size, num_pages};
    float* part_acc = scratch;
    float* part_ml = scratch ? scratch + static_cast<size_t>(n_rows) * nq * num_splits * dv : nullptr;
    cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
#define LAUNCH(DD)                                                                                                         \
    do {                                                                                                                      \
        auto kern = wide_decode_kernel<DD>;                                                                                \
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)); \
        if (e != cudaSuccess) return static_cast<int>(e);                                                                  \
        launch_pdl(kern, dim3(num_splits, nkv, n_rows), dim3(WD_THREADS), smem, s, static_cast<const bf16*>(q), c, rows,   \
                   positions, token_entry, entry_slot, block_table, table_stride, part_acc, part_ml, static_cast<bf16*>(out), nq, nkv, \
                   window, scale * 1.4426950408889634f, num_splits, status, out_scale, out_stride, out_off);               \
    } while (0)
    WIDE_BY_DV(LAUNCH)
#undef LAUNCH
    const int done = launch_status();
    if (done != LLM_OK || num_splits == 1) return done;
    launch_pdl(wide_combine_kernel, dim3(n_rows, nq), dim3(dv <= 64 ? 64 : 128), 0, s, part_acc, part_ml, rows, static_cast<bf16*>(out), nq,
               dv, num_splits, out_scale, out_stride, out_off);
    return launch_status();
}
