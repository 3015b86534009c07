// Device code of the tensor-core attention over the paged cache for bfloat16 models: one kernel for steps in which every
// sequence brings one token (keys split over blocks, partial results merged in a fixed order) and one for
// steps that bring many tokens per sequence (causal, blockwise with an online softmax).
//
// The formula is the reference's (src/minimax.rs:270-281): s = q.k * scale over the visible keys,
// p = softmax(s), out = p V, query head h reading kv head h / (heads / kv_heads).  Scores, the running
// maximum and sum, and both accumulators are float32; only the operands of the two products are bfloat16.
//
// Both kernels work on tiles of 16 rows x 64 keys (one cache page) held in registers.  Operands go from
// global memory straight into mma.sync fragments with 16-byte loads: a product over k does not depend on
// the order of k, so each thread takes 8 neighbouring elements of k for two MMAs instead of the scattered
// pairs of the fragment layout, on both operands alike.  Values lie transposed within a page
// ([head_dim][64 keys]), which makes the keys of P @ V neighbours in memory too.
#pragma once

#include "common.cuh"

#define ATT_CHUNK 256          // keys per block of the one-token kernel: 4 warps x 1 page

__device__ __forceinline__ void mma_bf16(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0,
                                         uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&v);
}

// A tile of 16 rows: lane = 4 g + t holds rows g and g + 8.
template <int HD, int VD>
struct RowTile {
    uint4 q[HD / 32][2];       // [32 dims][row g | row g+8]: dims 32 s + 8 t .. + 7
    float o[VD / 8][4];        // [8 value dims]: (row g, dims 8 n + 2t, +1), (row g+8, same dims)
    float m[2], l[2];          // running maximum (in units of log2) and sum of rows g and g + 8
};

template <int HD, int VD>
__device__ __forceinline__ void tile_init(RowTile<HD, VD>& st) {
#pragma unroll
    for (int n = 0; n < VD / 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) st.o[n][e] = 0.f;
    st.m[0] = st.m[1] = -INFINITY;
    st.l[0] = st.l[1] = 0.f;
}

// Where a page's operands are read from: global memory (the page itself) ...
template <int HD>
struct GlobalPage {
    const bf16* k_page;      // [64][HD]
    const bf16* vt_page;     // [VD][64]
    // 8 dims 32 step + 8 t .. of key `key`
    __device__ __forceinline__ uint4 k(int key, int step, int t) const {
        return __ldg(reinterpret_cast<const uint4*>(k_page + (size_t)key * HD) + step * 4 + t);
    }
    // 8 keys 32 m + 8 t .. of dim `dim`
    __device__ __forceinline__ uint4 v(int dim, int m, int t) const {
        return __ldg(reinterpret_cast<const uint4*>(vt_page + (size_t)dim * FRB_PAGE) + m * 4 + t);
    }
};

// ... or a copy of the page in shared memory, whose 16-byte chunks are swizzled so that the eight lanes of
// a quarter warp (two rows, four chunks each) fall into different banks: chunk ^= (row & 1) << 2, for the
// chunks that lie in whole groups of eight.
template <int CHUNKS_PER_ROW>
__device__ __forceinline__ int swizzled(int chunk, int row) {
    return chunk < (CHUNKS_PER_ROW & ~7) ? chunk ^ ((row & 1) << 2) : chunk;
}

template <int HD>
struct SharedPage {
    const uint4* k_tile;     // [64][HD / 8] chunks
    const uint4* vt_tile;    // [VD][8] chunks
    __device__ __forceinline__ uint4 k(int key, int step, int t) const {
        return k_tile[key * (HD / 8) + swizzled<HD / 8>(step * 4 + t, key)];
    }
    __device__ __forceinline__ uint4 v(int dim, int m, int t) const {
        return vt_tile[dim * 8 + swizzled<8>(m * 4 + t, dim)];
    }
};

// Adds one page of 64 keys to the tile.  key_base: position of the page's first key; row r sees keys
// lo[r] <= j <= hi[r].  scale2 = softmax scale * log2(e).  slope2 = the head's distance slope * log2(e): the score
// of key j for the query at position hi[r] is lowered by slope * (hi[r] - j); 0 for none.  Keys before keep_first are
// visible to every row that is not before them.
template <int HD, int VD, typename Page>
__device__ __forceinline__ void tile_page(RowTile<HD, VD>& st, const Page& page, int key_base, const int (&lo)[2],
                                          const int (&hi)[2], float scale2, int g, int t, float slope2 = 0.f,
                                          float cap_scale = 0.f, float cap2 = 0.f, int keep_first = 0) {
    float s[8][4];
    // scores: column block 4 m + u, column c = 2 t' + d of it stands for key 32 m + 8 t' + 2 u + d
#pragma unroll
    for (int m = 0; m < 2; ++m) {
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int key_local = 32 * m + 8 * (g >> 1) + 2 * u + (g & 1);
            float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int step = 0; step < HD / 32; ++step) {
                const uint4 kb = page.k(key_local, step, t);
                mma_bf16(acc, st.q[step][0].x, st.q[step][1].x, st.q[step][0].y, st.q[step][1].y, kb.x, kb.y);
                mma_bf16(acc, st.q[step][0].z, st.q[step][1].z, st.q[step][0].w, st.q[step][1].w, kb.z, kb.w);
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) s[4 * m + u][e] = acc[e];
        }
    }
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int m = 0; m < 2; ++m)
#pragma unroll
        for (int u = 0; u < 4; ++u)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int r = e >> 1;
                const int key = key_base + 32 * m + 8 * t + 2 * u + (e & 1);
                const float raw = s[4 * m + u][e];
                const float scaled = cap2 > 0.f ? capped_score2(raw, cap_scale, cap2) : raw * scale2;
                const float v = key_visible(key, lo[r], hi[r], keep_first) ? fmaf(slope2, (float)(key - hi[r]), scaled) : -INFINITY;
                s[4 * m + u][e] = v;
                mx[r] = fmaxf(mx[r], v);
            }
    float corr[2], sum[2] = {0.f, 0.f}, m_use[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
        const float m_new = fmaxf(st.m[r], mx[r]);
        m_use[r] = (m_new == -INFINITY) ? 0.f : m_new;       // a row that has seen no key yet
        corr[r] = exp2f(st.m[r] - m_use[r]);
        st.m[r] = m_new;
    }
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const float pv = exp2f(s[j][e] - m_use[e >> 1]);
            s[j][e] = pv;
            sum[e >> 1] += pv;
        }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 1);
        sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 2);
        st.l[r] = st.l[r] * corr[r] + sum[r];
    }
#pragma unroll
    for (int n = 0; n < VD / 8; ++n) {
        st.o[n][0] *= corr[0]; st.o[n][1] *= corr[0];
        st.o[n][2] *= corr[1]; st.o[n][3] *= corr[1];
    }
    // out += P V: the thread's 8 keys 32 m + 8 t .. + 7 are one 16-byte run of a transposed value row
#pragma unroll
    for (int m = 0; m < 2; ++m) {
        const uint32_t a0 = pack_bf16(s[4 * m][0], s[4 * m][1]), a1 = pack_bf16(s[4 * m][2], s[4 * m][3]);
        const uint32_t a2 = pack_bf16(s[4 * m + 1][0], s[4 * m + 1][1]), a3 = pack_bf16(s[4 * m + 1][2], s[4 * m + 1][3]);
        const uint32_t b0 = pack_bf16(s[4 * m + 2][0], s[4 * m + 2][1]), b1 = pack_bf16(s[4 * m + 2][2], s[4 * m + 2][3]);
        const uint32_t b2 = pack_bf16(s[4 * m + 3][0], s[4 * m + 3][1]), b3 = pack_bf16(s[4 * m + 3][2], s[4 * m + 3][3]);
#pragma unroll
        for (int n = 0; n < VD / 8; ++n) {
            const uint4 vb = page.v(8 * n + g, m, t);
            mma_bf16(st.o[n], a0, a1, a2, a3, vb.x, vb.y);
            mma_bf16(st.o[n], b0, b1, b2, b3, vb.z, vb.w);
        }
    }
}

template <int HD, int VD>
__device__ __forceinline__ void load_q_row(RowTile<HD, VD>& st, int half, const bf16* __restrict__ row, int t) {
#pragma unroll
    for (int step = 0; step < HD / 32; ++step)
        st.q[step][half] = row ? __ldg(reinterpret_cast<const uint4*>(row + 32 * step) + t) : make_uint4(0, 0, 0, 0);
}

// ----------------------------------------------------------------------------- one token per sequence

struct DecodeAttnParams {
    const bf16* q;             // [B, nh, HD]
    const bf16* k_pages;       // [pages, nkv, 64, HD]
    const bf16* v_pages;       // [pages, v_heads, VD, 64]
    const int* page_table;     // [slots, max_pages]
    const int* seq_pos;        // [B] position of the sequence's token
    const int* seq_slot;       // [B]
    float* part_o;             // [B, nh, max_chunks, VD]
    float* part_ml;            // [B, nh, max_chunks, 2]
    bf16* out;                 // [B, nh * VD], or with two maps per head [B, nh / 2 * VD]
    float scale2;
    int window, max_pages, num_heads, num_kv_heads, max_chunks;
    int* status;               // null, or a word that gets FRB_STATUS_TOO_LONG when a sequence has more chunks than max_chunks
    const float* slopes;       // null, or one slope per query head: key j's score is lowered by slope * (position - j)
    int chunk;                 // 0, or the token sees only the keys of its own chunk of this many positions
    const float* sinks;        // null, or one number per query head whose exponential joins the softmax's denominator
    float cap_scale, cap2;     // capped scores (capped_score2): scale / cap and cap * log2(e); cap2 0: none
    int keep_first;            // with a window: the sequence's first tokens that stay visible beside it
    int v_heads;               // value heads; key heads in runs of num_kv_heads / v_heads share one
    // Two maps per head (lam not null): query heads lie as [value head, map, query head of the group], and the output of a
    // head is o / sqrt(mean(o^2) + diff_eps) * diff_factor with o = map 1 - lam * map 2, taken where partial results are joined.
    const float* lam;
    float diff_eps, diff_factor;
};

// What the entry points take beyond the sizes that every call has (zero and null: off).
struct AttnExtras {
    const float* slopes = nullptr;
    int chunk = 0;
    const float* sinks = nullptr;
    float softcap = 0.f;
    int v_dim = 0, keep_first = 0, v_heads = 0;
    const float* lam = nullptr;
    float diff_eps = 0.f, diff_factor = 0.f;
};

// The slopes of the two query heads that a thread's rows g and g + 8 of the group's tile stand for, times log2(e).
__device__ __forceinline__ void group_slopes(const float* slopes, int first_head, int group, int g, float (&slope2)[2]) {
    slope2[0] = (slopes && g < group) ? slopes[first_head + g] * 1.4426950408889634f : 0.f;
    slope2[1] = (slopes && g + 8 < group) ? slopes[first_head + g + 8] * 1.4426950408889634f : 0.f;
}

#define FRB_STATUS_TOO_LONG 5

// grid (chunk, kv head, sequence), 4 warps.  Rows of the tile are the query heads of the kv head's group.
// Each warp takes one page of the chunk: scores, softmax within the page, then P V in two halves of the
// head size so that few accumulators are alive at a time (more blocks per SM, more loads in flight); the
// four warps' results are combined through shared memory.
template <int HD, int VD>
__global__ void __launch_bounds__(128, 4) attention_decode_mma_kernel(DecodeAttnParams p) {
    after_previous_kernel();
    __shared__ float sm_o[4][16][VD + 8];
    __shared__ float sm_m[4][16], sm_l[4][16];
    const int chunk = blockIdx.x, kvh = blockIdx.y, b = blockIdx.z;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
    const int group = p.num_heads / p.num_kv_heads;
    const int pos = p.seq_pos[b];
    const int hi_key = pos, lo_key = first_visible_key(pos, p.window, p.chunk);
    if (chunk * ATT_CHUNK > hi_key || ((chunk + 1) * ATT_CHUNK <= lo_key && chunk * ATT_CHUNK >= p.keep_first))
        return;                                                                       // the merge skips these chunks

    const int page_index = chunk * (ATT_CHUNK / FRB_PAGE) + warp;
    const int key_base = page_index * FRB_PAGE;
    float row_max[2] = {-INFINITY, -INFINITY}, row_sum[2] = {0.f, 0.f};
    if (key_base <= hi_key && (key_base + FRB_PAGE > lo_key || key_base < p.keep_first)) {
        const int page = p.page_table[(size_t)p.seq_slot[b] * p.max_pages + page_index];
        const size_t at = ((size_t)page * p.num_kv_heads + kvh) * FRB_PAGE * HD;
        const int vh = kvh / (p.num_kv_heads / p.v_heads);
        const GlobalPage<HD> operands = {p.k_pages + at, p.v_pages + ((size_t)page * p.v_heads + vh) * FRB_PAGE * VD};
        float s[8][4];
        float slope2[2];
        group_slopes(p.slopes, kvh * group, group, g, slope2);
        {
            const bf16* q_base = p.q + ((size_t)b * p.num_heads + (size_t)kvh * group) * HD;
            const bf16* q0 = g < group ? q_base + (size_t)g * HD : nullptr;
            const bf16* q1 = g + 8 < group ? q_base + (size_t)(g + 8) * HD : nullptr;
            uint4 q[HD / 32][2];
#pragma unroll
            for (int step = 0; step < HD / 32; ++step) {
                q[step][0] = q0 ? __ldg(reinterpret_cast<const uint4*>(q0 + 32 * step) + t) : make_uint4(0, 0, 0, 0);
                q[step][1] = q1 ? __ldg(reinterpret_cast<const uint4*>(q1 + 32 * step) + t) : make_uint4(0, 0, 0, 0);
            }
#pragma unroll
            for (int m = 0; m < 2; ++m)
#pragma unroll
                for (int u = 0; u < 4; ++u) {
                    const int key_local = 32 * m + 8 * (g >> 1) + 2 * u + (g & 1);
                    float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                    for (int step = 0; step < HD / 32; ++step) {
                        const uint4 kb = operands.k(key_local, step, t);
                        mma_bf16(acc, q[step][0].x, q[step][1].x, q[step][0].y, q[step][1].y, kb.x, kb.y);
                        mma_bf16(acc, q[step][0].z, q[step][1].z, q[step][0].w, q[step][1].w, kb.z, kb.w);
                    }
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int key = key_base + 32 * m + 8 * t + 2 * u + (e & 1);
                        const float scaled = p.cap2 > 0.f ? capped_score2(acc[e], p.cap_scale, p.cap2) : acc[e] * p.scale2;
                        const float v = key_visible(key, lo_key, hi_key, p.keep_first) ? fmaf(slope2[e >> 1], (float)(key - hi_key), scaled) : -INFINITY;
                        s[4 * m + u][e] = v;
                        row_max[e >> 1] = fmaxf(row_max[e >> 1], v);
                    }
                }
        }
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            row_max[r] = fmaxf(row_max[r], __shfl_xor_sync(0xffffffffu, row_max[r], 1));
            row_max[r] = fmaxf(row_max[r], __shfl_xor_sync(0xffffffffu, row_max[r], 2));
        }
        // the page holds at least one visible key, and every row sees the same keys: the maxima are finite
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float pv = exp2f(s[j][e] - row_max[e >> 1]);
                s[j][e] = pv;
                row_sum[e >> 1] += pv;
            }
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            row_sum[r] += __shfl_xor_sync(0xffffffffu, row_sum[r], 1);
            row_sum[r] += __shfl_xor_sync(0xffffffffu, row_sum[r], 2);
        }
        uint32_t pa[2][4], pb[2][4];
#pragma unroll
        for (int m = 0; m < 2; ++m) {
            pa[m][0] = pack_bf16(s[4 * m][0], s[4 * m][1]);         pa[m][1] = pack_bf16(s[4 * m][2], s[4 * m][3]);
            pa[m][2] = pack_bf16(s[4 * m + 1][0], s[4 * m + 1][1]); pa[m][3] = pack_bf16(s[4 * m + 1][2], s[4 * m + 1][3]);
            pb[m][0] = pack_bf16(s[4 * m + 2][0], s[4 * m + 2][1]); pb[m][1] = pack_bf16(s[4 * m + 2][2], s[4 * m + 2][3]);
            pb[m][2] = pack_bf16(s[4 * m + 3][0], s[4 * m + 3][1]); pb[m][3] = pack_bf16(s[4 * m + 3][2], s[4 * m + 3][3]);
        }
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            float o[VD / 16][4];
#pragma unroll
            for (int n = 0; n < VD / 16; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) o[n][e] = 0.f;
#pragma unroll
            for (int m = 0; m < 2; ++m)
#pragma unroll
                for (int n = 0; n < VD / 16; ++n) {
                    const uint4 vb = operands.v(8 * (half * (VD / 16) + n) + g, m, t);
                    mma_bf16(o[n], pa[m][0], pa[m][1], pa[m][2], pa[m][3], vb.x, vb.y);
                    mma_bf16(o[n], pb[m][0], pb[m][1], pb[m][2], pb[m][3], vb.z, vb.w);
                }
#pragma unroll
            for (int n = 0; n < VD / 16; ++n) {
                const int d = 8 * (half * (VD / 16) + n) + 2 * t;
                *reinterpret_cast<float2*>(&sm_o[warp][g][d]) = make_float2(o[n][0], o[n][1]);
                *reinterpret_cast<float2*>(&sm_o[warp][g + 8][d]) = make_float2(o[n][2], o[n][3]);
            }
        }
    }
    if (t == 0) {
        sm_m[warp][g] = row_max[0]; sm_l[warp][g] = row_sum[0];
        sm_m[warp][g + 8] = row_max[1]; sm_l[warp][g + 8] = row_sum[1];
    }
    __syncthreads();
    for (int idx = threadIdx.x; idx < group * VD; idx += 128) {
        const int r = idx / VD, d = idx - r * VD;
        float top = -INFINITY;
#pragma unroll
        for (int w = 0; w < 4; ++w) top = fmaxf(top, sm_m[w][r]);
        float sum = 0.f, acc = 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w) {
            if (sm_l[w][r] > 0.f) {                             // a warp whose page holds no visible key wrote nothing
                const float f = exp2f(sm_m[w][r] - top);
                sum += sm_l[w][r] * f;
                acc += sm_o[w][r][d] * f;
            }
        }
        const size_t row = ((size_t)b * p.num_heads + (size_t)kvh * group + r) * p.max_chunks + chunk;
        p.part_o[row * VD + d] = acc;
        if (d == 0) { p.part_ml[row * 2] = top; p.part_ml[row * 2 + 1] = sum; }
    }
}

// Element d of the merged output of one (sequence, head) from the partial results 0 .. kept - 1, then first .. last
// (maximum and sum in part_ml, unnormalised output in part_o), in that order.  Eight results at a time, all of their loads
// asked for before the first is used: in a plain loop over the results each load waited for the one before it, which was
// most of the merge's time.
template <int VD>
__device__ __forceinline__ float merged_element(const float* __restrict__ part_ml, const float* __restrict__ part_o, size_t row0,
                                                int kept, int first, int last, int d, float sink2 = -INFINITY) {
    constexpr int AT_ONCE = 8;
    float top = -INFINITY, sum = 0.f, acc = 0.f;
    const int end = kept + last - first;                  // the last result's number
    for (int c0 = 0; c0 <= end; c0 += AT_ONCE) {
        float2 ml[AT_ONCE];
        float o[AT_ONCE];
#pragma unroll
        for (int u = 0; u < AT_ONCE; ++u) {
            const int c = run_at(min(c0 + u, end), kept, first);
            ml[u] = *reinterpret_cast<const float2*>(part_ml + (row0 + c) * 2);
            o[u] = part_o[(row0 + c) * VD + d];
        }
        float group_top = top;
#pragma unroll
        for (int u = 0; u < AT_ONCE; ++u)
            if (c0 + u <= end) group_top = fmaxf(group_top, ml[u].x);
        // what was summed so far follows the new maximum (nothing was summed before the first group)
        const float keep = top == -INFINITY ? 0.f : exp2f(top - group_top);
        sum *= keep;
        acc *= keep;
        top = group_top;
#pragma unroll
        for (int u = 0; u < AT_ONCE; ++u)
            if (c0 + u <= end) {
                const float f = exp2f(ml[u].x - top);
                sum += ml[u].y * f;
                acc += o[u] * f;
            }
    }
    if (sink2 > -INFINITY) {                              // a sink: a term of the denominator without a value (log2 units)
        const float top_all = fmaxf(top, sink2);
        const float keep = exp2f(top - top_all);
        sum = sum * keep + exp2f(sink2 - top_all);
        acc *= keep;
    }
    return acc / sum;
}

// The joined output of one head, a thread per value entry (blockDim.x = VD); grid (output head, sequence).  With two maps per
// head both are joined, and their difference is normed over the block.
template <int VD>
__device__ __forceinline__ void merge_head(const DecodeAttnParams& p, int keys_per_part, int* status) {
    __shared__ float scratch[32];
    const int head = blockIdx.x, b = blockIdx.y, d = threadIdx.x;
    const int pos = p.seq_pos[b];
    const int lo_key = first_visible_key(pos, p.window, p.chunk);
    // never beyond the partial results the launch has room for, whatever the position says (the caller's
    // max_chunks covers the longest sequence; a smaller one must not make this read another row's results)
    const int last = min(pos / keys_per_part, p.max_chunks - 1), first = min(lo_key / keys_per_part, last);
    const int kept = kept_runs(p.keep_first, keys_per_part, first);
    if (pos / keys_per_part >= p.max_chunks && status && d == 0) atomicExch(status, FRB_STATUS_TOO_LONG);   // keys were left out
    if (p.lam) {
        const int group = p.num_heads / p.num_kv_heads, g = head / group, heads = p.num_heads / 2;
        const size_t row1 = ((size_t)b * p.num_heads + (size_t)(2 * g) * group + (head - g * group)) * p.max_chunks;
        const size_t row2 = row1 + (size_t)group * p.max_chunks;
        const float a1 = merged_element<VD>(p.part_ml, p.part_o, row1, kept, first, last, d);
        const float a2 = merged_element<VD>(p.part_ml, p.part_o, row2, kept, first, last, d);
        const float o = a1 - *p.lam * a2;
        const float ss = block_sum<VD>(o * o, scratch);
        p.out[((size_t)b * heads + head) * VD + d] = __float2bfloat16_rn(o / sqrtf(ss / (float)VD + p.diff_eps) * p.diff_factor);
        return;
    }
    const size_t row0 = ((size_t)b * p.num_heads + head) * p.max_chunks;
    p.out[((size_t)b * p.num_heads + head) * VD + d] = __float2bfloat16_rn(merged_element<VD>(
        p.part_ml, p.part_o, row0, kept, first, last, d, p.sinks ? p.sinks[head] * 1.4426950408889634f : -INFINITY));
}

// grid (head, sequence): merges the chunks of one (sequence, head), first chunk to last.
template <int VD>
__global__ void __launch_bounds__(VD) attention_decode_merge_kernel(DecodeAttnParams p) {
    after_previous_kernel();
    merge_head<VD>(p, ATT_CHUNK, p.status);
}

// Fills what the one-token kernels share; -1 if sizes do not fit together.
static inline int fill_decode_extras(const char* what, DecodeAttnParams& p, int head_dim, float scale, const AttnExtras& x) {
    p.slopes = x.slopes; p.chunk = x.chunk; p.sinks = x.sinks;
    p.cap_scale = x.softcap > 0.f ? scale / x.softcap : 0.f; p.cap2 = x.softcap > 0.f ? x.softcap * 1.4426950408889634f : 0.f;
    p.keep_first = p.window > 0 ? x.keep_first : 0;
    p.v_heads = x.v_heads > 0 ? x.v_heads : p.num_kv_heads;
    p.lam = x.lam; p.diff_eps = x.diff_eps; p.diff_factor = x.diff_factor;
    FRB_CHECK_ARG(x.keep_first >= 0 && !(x.keep_first > 0 && x.chunk > 0), "%s: %d first tokens together with chunks", what, x.keep_first);
    FRB_CHECK_ARG(p.num_kv_heads % p.v_heads == 0, "%s: %d key heads over %d value heads", what, p.num_kv_heads, p.v_heads);
    FRB_CHECK_ARG(!x.lam || (p.num_kv_heads == 2 * p.v_heads && !x.sinks), "%s: two maps per head need two key heads a value head and no sinks", what);
    return 0;
}

// Calls LAUNCH(HD, VD) with the head sizes as constants: key and value heads of one size, or value heads twice the key heads.
#define FRB_ATTENTION_SIZES(head_dim, v_dim, LAUNCH)                                             \
    do {                                                                                         \
        if (head_dim == 32 && v_dim == 32) { LAUNCH(32, 32); }                                   \
        else if (head_dim == 32) { LAUNCH(32, 64); }                                             \
        else if (head_dim == 64 && v_dim == 64) { LAUNCH(64, 64); }                              \
        else if (head_dim == 64) { LAUNCH(64, 128); }                                            \
        else if (head_dim == 96) { LAUNCH(96, 96); }                                             \
        else { LAUNCH(128, 128); }                                                               \
    } while (0)

static inline bool attention_sizes_built(int head_dim, int v_dim) {
    const bool same = head_dim == v_dim && (head_dim == 32 || head_dim == 64 || head_dim == 96 || head_dim == 128);
    return same || (v_dim == 2 * head_dim && (head_dim == 32 || head_dim == 64));
}

// Checks the sizes and launches the one-token kernel and its merge.  `what` names the caller in errors.
static inline int launch_attention_decode(const char* what, const void* q, const void* k_pages, const void* v_pages,
                                          const int* page_table, int max_pages, const int* seq_pos, const int* seq_slot,
                                          float* part_o, float* part_ml, void* out, int num_seqs, int num_heads,
                                          int num_kv_heads, int head_dim, float scale, int window, int max_chunks,
                                          cudaStream_t stream, int* status = nullptr, const AttnExtras& extras = AttnExtras()) {
    if (num_seqs == 0) return 0;
    const int v_dim = extras.v_dim > 0 ? extras.v_dim : head_dim;
    const int group = num_kv_heads > 0 ? num_heads / num_kv_heads : 0;
    FRB_CHECK_ARG(num_kv_heads > 0 && num_heads % num_kv_heads == 0 && group <= 16,
                  "%s: %d heads over %d kv heads (groups of at most 16)", what, num_heads, num_kv_heads);
    FRB_CHECK_ARG(attention_sizes_built(head_dim, v_dim), "%s: head_dim %d with value heads of %d is not built", what, head_dim, v_dim);
    FRB_CHECK_ARG(num_seqs <= 65535 && num_kv_heads <= 65535, "%s: %d sequences exceed the grid", what, num_seqs);
    DecodeAttnParams p;
    p.q = (const bf16*)q; p.k_pages = (const bf16*)k_pages; p.v_pages = (const bf16*)v_pages; p.page_table = page_table;
    p.seq_pos = seq_pos; p.seq_slot = seq_slot; p.part_o = part_o; p.part_ml = part_ml; p.out = (bf16*)out;
    p.scale2 = scale * 1.4426950408889634f; p.window = window; p.max_pages = max_pages; p.num_heads = num_heads;
    p.num_kv_heads = num_kv_heads; p.max_chunks = max_chunks; p.status = status;
    if (fill_decode_extras(what, p, head_dim, scale, extras)) return -1;
    dim3 grid(max_chunks, num_kv_heads, num_seqs), merge_grid(extras.lam ? num_heads / 2 : num_heads, num_seqs);
#define FRB_LAUNCH_DECODE(HD, VD)                                                                              \
    launch_dependent(attention_decode_mma_kernel<HD, VD>, dim3(grid), dim3(128), 0, stream, p);                \
    launch_dependent(attention_decode_merge_kernel<VD>, dim3(merge_grid), dim3(VD), 0, stream, p)
    FRB_ATTENTION_SIZES(head_dim, v_dim, FRB_LAUNCH_DECODE);
#undef FRB_LAUNCH_DECODE
    FRB_RETURN_LAUNCH(what);
}
