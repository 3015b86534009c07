// Entry points of the tensor-core attention (bfloat16): steps of one token per sequence, and steps of many.
// The kernels are in attention_mma.cuh.
#include "attention_mma.cuh"

FRB_API int frb_attention_decode_mma(const void* q, const void* k_pages, const void* v_pages, const int* page_table,
                                     int max_pages, const int* seq_pos, const int* seq_slot, float* part_o, float* part_ml,
                                     void* out, int num_seqs, int num_heads, int num_kv_heads, int head_dim, float scale,
                                     int window, int max_chunks, int* status, const float* slopes, int chunk, const float* sinks,
                                     float softcap, int v_dim, int keep_first, int v_heads, const float* lam, float diff_eps,
                                     float diff_factor, cudaStream_t stream) {
    AttnExtras extras;
    extras.slopes = slopes; extras.chunk = chunk; extras.sinks = sinks; extras.softcap = softcap; extras.v_dim = v_dim;
    extras.keep_first = keep_first; extras.v_heads = v_heads; extras.lam = lam; extras.diff_eps = diff_eps; extras.diff_factor = diff_factor;
    return launch_attention_decode("attention_decode_mma", q, k_pages, v_pages, page_table, max_pages, seq_pos, seq_slot,
                                   part_o, part_ml, out, num_seqs, num_heads, num_kv_heads, head_dim, scale, window,
                                   max_chunks, stream, status, extras);
}

// ----------------------------------------------------------------------------- many tokens per sequence

struct PrefillAttnParams {
    const bf16* q;             // [T, nh, HD]
    const bf16* k_pages;
    const bf16* v_pages;
    const int* page_table;
    const int* tile_seq;       // [tiles] sequence of the tile
    const int* tile_q0;        // [tiles] first row of the tile among its sequence's new tokens
    const int* seq_slot;       // [B]
    const int* seq_start;      // [B] position of the sequence's first new token
    const int* seq_q_len;      // [B]
    const int* cu_q_len;       // [B + 1]
    bf16* out;                 // [T, nh * VD]
    float* out32;              // null, or the output in float32 instead
    float scale2;
    int window, max_pages, num_heads, num_kv_heads;
    const float* slopes;       // null, or one slope per query head: key j's score is lowered by slope * (position - j)
    int chunk;                 // 0, or a query sees only the keys of its own chunk of this many positions
    const float* sinks;        // null, or one number per query head whose exponential joins the softmax's denominator
    float cap_scale, cap2;     // capped scores (capped_score2): scale / cap and cap * log2(e); cap2 0: none
    int keep_first, v_heads;   // first tokens that stay visible beside the window; value heads (runs of key heads share one)
};

__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

// Starts the copy of one page's keys and transposed values into a stage of shared memory (swizzled chunks).
template <int HD, int VD>
__device__ __forceinline__ void stage_page(uint4* k_tile, uint4* vt_tile, const bf16* __restrict__ k_page,
                                           const bf16* __restrict__ vt_page) {
    for (int c = threadIdx.x; c < FRB_PAGE * HD / 8; c += blockDim.x) {       // 16-byte chunks of K
        const int key = c / (HD / 8), chunk = c % (HD / 8);
        cp_async16(k_tile + key * (HD / 8) + swizzled<HD / 8>(chunk, key), reinterpret_cast<const uint4*>(k_page) + c);
    }
    for (int c = threadIdx.x; c < FRB_PAGE * VD / 8; c += blockDim.x) {       // and of V
        const int dim = c >> 3, vchunk = c & 7;
        cp_async16(vt_tile + dim * 8 + swizzled<8>(vchunk, dim), reinterpret_cast<const uint4*>(vt_page) + c);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
}

// grid (tile of 16 queries, kv head).  The warps of a block take the query heads of the kv head's group:
// they need the same keys and values, which the block copies page by page into two stages of shared memory
// with cp.async, the next page on its way while the current one is multiplied.
template <int HD, int VD, int MAX_WARPS>
__global__ void __launch_bounds__(MAX_WARPS * 32, MAX_WARPS <= 6 ? 2 : 1) attention_prefill_mma_kernel(PrefillAttnParams p) {
    extern __shared__ uint4 stages[];                   // 2 x (K tile, V^T tile)
    constexpr int K_TILE = FRB_PAGE * HD / 8, STAGE = K_TILE + FRB_PAGE * VD / 8;      // 16-byte chunks
    const int tile = blockIdx.x, kvh = blockIdx.y;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5, g = lane >> 2, t = lane & 3;
    const int group = p.num_heads / p.num_kv_heads;
    const int b = p.tile_seq[tile], q0 = p.tile_q0[tile];
    const int q_len = p.seq_q_len[b], start = p.seq_start[b], tok0 = p.cu_q_len[b] + q0;
    const int* table = p.page_table + (size_t)p.seq_slot[b] * p.max_pages;
    int lo[2], hi[2];
    bool valid[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const int row = g + 8 * r;
        valid[r] = q0 + row < q_len;
        hi[r] = valid[r] ? start + q0 + row : -1;
        lo[r] = valid[r] ? first_visible_key(hi[r], p.window, p.chunk) : 0;
    }
    const int last_key = start + min(q0 + 15, q_len - 1);
    const int first_key = first_visible_key(start + q0, p.window, p.chunk);
    // the pages of the first tokens that stay visible, then those from the window on
    const int first_page = first_key / FRB_PAGE, kept = kept_runs(p.keep_first, FRB_PAGE, first_page);
    const int num_pages = kept + last_key / FRB_PAGE - first_page + 1;
    const int vh = kvh / (p.num_kv_heads / p.v_heads);
    auto stage = [&](int n) {
        const int page = table[run_at(n, kept, first_page)];
        uint4* at = stages + (n & 1) * STAGE;
        stage_page<HD, VD>(at, at + K_TILE, p.k_pages + ((size_t)page * p.num_kv_heads + kvh) * FRB_PAGE * HD,
                           p.v_pages + ((size_t)page * p.v_heads + vh) * FRB_PAGE * VD);
    };
    for (int hbase = 0; hbase < group; hbase += nwarps) {
        const int hl = hbase + warp;
        const bool active = hl < group;
        const int head = kvh * group + (active ? hl : 0);
        RowTile<HD, VD> st;
        tile_init(st);
        const float slope2 = p.slopes ? p.slopes[head] * 1.4426950408889634f : 0.f;
#pragma unroll
        for (int r = 0; r < 2; ++r)
            load_q_row(st, r, (active && valid[r]) ? p.q + ((size_t)(tok0 + g + 8 * r) * p.num_heads + head) * HD : nullptr, t);
        stage(0);
        for (int n = 0; n < num_pages; ++n) {
            if (n + 1 < num_pages) {
                stage(n + 1);
                asm volatile("cp.async.wait_group 1;" ::: "memory");
            } else {
                asm volatile("cp.async.wait_group 0;" ::: "memory");
            }
            __syncthreads();
            if (active) {
                const SharedPage<HD> page = {stages + (n & 1) * STAGE, stages + (n & 1) * STAGE + K_TILE};
                tile_page(st, page, run_at(n, kept, first_page) * FRB_PAGE, lo, hi, p.scale2, g, t, slope2, p.cap_scale, p.cap2,
                          p.keep_first);
            }
            __syncthreads();                            // the stage is free for the page after the next
        }
        if (active) {
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                if (!valid[r]) continue;
                float scale_o = 1.f, total = st.l[r];
                if (p.sinks) {                              // the sink joins the denominator (log2 units, like st.m)
                    const float sink2 = p.sinks[head] * 1.4426950408889634f, top = fmaxf(st.m[r], sink2);
                    scale_o = exp2f(st.m[r] - top);
                    total = total * scale_o + exp2f(sink2 - top);
                }
                const float inv = scale_o / total;
                const size_t dst = ((size_t)(tok0 + g + 8 * r) * p.num_heads + head) * VD;
#pragma unroll
                for (int n = 0; n < VD / 8; ++n) {
                    const float a = st.o[n][2 * r] * inv, c = st.o[n][2 * r + 1] * inv;
                    if (p.out32) *reinterpret_cast<float2*>(p.out32 + dst + 8 * n + 2 * t) = make_float2(a, c);
                    else *reinterpret_cast<uint32_t*>(p.out + dst + 8 * n + 2 * t) = pack_bf16(a, c);
                }
            }
        }
    }
}

FRB_API int frb_attention_prefill_mma(const void* q, const void* k_pages, const void* v_pages, const int* page_table,
                                      int max_pages, const int* tile_seq, const int* tile_q0, int num_tiles,
                                      const int* seq_slot, const int* seq_start, const int* seq_q_len, const int* cu_q_len,
                                      void* out, int num_heads, int num_kv_heads, int head_dim, float scale, int window,
                                      const float* slopes, int chunk, const float* sinks, float softcap, int v_dim, int keep_first,
                                      int v_heads, int out_f32, cudaStream_t stream) {
    if (num_tiles == 0) return 0;
    if (v_dim <= 0) v_dim = head_dim;
    if (v_heads <= 0) v_heads = num_kv_heads;
    FRB_CHECK_ARG(num_kv_heads > 0 && num_heads % num_kv_heads == 0, "attention: %d heads over %d kv heads", num_heads, num_kv_heads);
    FRB_CHECK_ARG(attention_sizes_built(head_dim, v_dim), "attention: head_dim %d with value heads of %d is not built", head_dim, v_dim);
    FRB_CHECK_ARG(num_kv_heads % v_heads == 0, "attention: %d key heads over %d value heads", num_kv_heads, v_heads);
    FRB_CHECK_ARG(keep_first >= 0 && !(keep_first > 0 && chunk > 0), "attention: %d first tokens together with chunks", keep_first);
    FRB_CHECK_ARG(num_kv_heads <= 65535, "attention: %d kv heads exceed the grid", num_kv_heads);
    PrefillAttnParams p;
    p.q = (const bf16*)q; p.k_pages = (const bf16*)k_pages; p.v_pages = (const bf16*)v_pages; p.page_table = page_table;
    p.tile_seq = tile_seq; p.tile_q0 = tile_q0; p.seq_slot = seq_slot; p.seq_start = seq_start; p.seq_q_len = seq_q_len;
    p.cu_q_len = cu_q_len; p.out = (bf16*)out; p.out32 = out_f32 ? (float*)out : nullptr;
    p.keep_first = window > 0 ? keep_first : 0; p.v_heads = v_heads; p.scale2 = scale * 1.4426950408889634f; p.window = window;
    p.max_pages = max_pages; p.num_heads = num_heads; p.num_kv_heads = num_kv_heads; p.slopes = slopes;
    p.chunk = chunk; p.sinks = sinks;
    p.cap_scale = softcap > 0.f ? scale / softcap : 0.f; p.cap2 = softcap > 0.f ? softcap * 1.4426950408889634f : 0.f;
    const int group = num_heads / num_kv_heads;
    const int nwarps = group < 8 ? group : 8;
    dim3 grid(num_tiles, num_kv_heads);
    const size_t smem = (size_t)2 * FRB_PAGE * (head_dim + v_dim) * sizeof(bf16);           // two stages of K and V^T
    // groups of up to 6 heads: blocks of at most 192 threads, held to two per SM; larger groups: 256 threads
#define LAUNCH(HD, VD)                                                                                              \
    if (nwarps <= 6) {                                                                                              \
        if (smem > 48 * 1024)                                                                                       \
            cudaFuncSetAttribute(attention_prefill_mma_kernel<HD, VD, 6>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        attention_prefill_mma_kernel<HD, VD, 6><<<grid, 32 * nwarps, smem, stream>>>(p);                            \
    } else {                                                                                                        \
        if (smem > 48 * 1024)                                                                                       \
            cudaFuncSetAttribute(attention_prefill_mma_kernel<HD, VD, 8>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        attention_prefill_mma_kernel<HD, VD, 8><<<grid, 32 * nwarps, smem, stream>>>(p);                            \
    }
    FRB_ATTENTION_SIZES(head_dim, v_dim, LAUNCH);
#undef LAUNCH
    FRB_RETURN_LAUNCH("attention_prefill_mma");
}
