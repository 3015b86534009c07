// Prompt attention with two maps per head on the fifth-generation tensor cores (tcgen05): both maps of a head, their
// difference and its norm in one kernel.
//
//   a_m = softmax(q_m k_m^T * scale, capped, masked) v,   o = a_1 - lam a_2,   out = o / sqrt(mean(o^2) + eps) * factor
//
// A block takes 128 queries of one head: two query tiles (a tile per map), and for every step of two cache pages (128 keys)
// the keys of both maps and one copy of the values that they share.
//   S_m = Q_m K_m^T   tcgen05.mma 128 x 128 x HD, a buffer of 128 columns of tensor memory per map;
//   softmax           eight warps, four per map, a thread per (map, query row) that takes all 128 keys of a step: the largest
//                     score first, then page by page the weights, written as bfloat16 over the columns of their scores;
//   O_m += P_m V      tcgen05.mma 128 x VD x 64 for each page, P_m as the tensor-memory operand.
// The maps take turns on the tensor core: while one map's softmax runs, the other's P V and next scores are computed.  The MMAs
// of the issuing thread run in the order of their issue, so S_m of step j + 1 goes into the buffer of step j right behind
// P_m V of step j, which reads it; and when S_m of a step has arrived, P_m V of the step before has ended, so O_m may be rescaled
// then.  At the end the two threads of a row exchange what they know of their maps, each takes half of the value entries of
// both, and the difference is normed and rounded once.
//
// The running maximum is raised lazily and every wait is bounded, as in attention_tc.cu.
#include "attention_tc.cuh"

#define AP_THREADS 320         // warp 0: TMA producer, warp 1: MMA issuer and tensor-memory owner, warps 2-5: map 1, 6-9: map 2
#define AP_SOFTMAX_THREADS 256
#define AP_STAGES 2
#define AP_STEP_PAGES 2
#define AP_STEP_KEYS (AP_STEP_PAGES * FRB_PAGE)

using namespace frb_tma;
using namespace frb_tc;
using namespace frb_at;

struct AttnPairParams {
    const int* page_table;
    const int* tile_seq;       // [tiles]
    const int* tile_q0;        // [tiles] first row of the tile among its sequence's new tokens
    const int* seq_slot;
    const int* seq_start;
    const int* seq_q_len;
    const int* cu_q_len;
    bf16* out;                 // [T, heads * VD]
    const float* lam;
    int* status;
    float scale2;              // softmax scale * log2(e)
    float cap_scale, cap2;     // CAPPED kernels (cap_scores): scale / cap and cap * log2(e)
    float eps, factor;
    int window, keep_first, max_pages, heads, v_heads;
};

// grid (tile of 128 queries, head); the longest tiles of a sequence (its last ones) start first.  Queries [T, v_heads, 2, group,
// HD], keys [pages, v_heads, 2, 64, HD], values [pages, v_heads, VD, 64].
template <int HD, int VD, bool CAPPED>
__global__ void __launch_bounds__(AP_THREADS)
attention_pair_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                         const __grid_constant__ CUtensorMap map_v, AttnPairParams p) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ uint64_t q_full, kv_full[AP_STAGES], kv_empty[AP_STAGES], s_full[2], p_full[2][AP_STEP_PAGES];
    __shared__ uint32_t tmem_slot;
    __shared__ int failed_flag;
    volatile int* failed = &failed_flag;
    static_assert(HD == 64 && VD <= 128, "tiles of one 128-byte row per key and query");
    constexpr uint32_t Q_BYTES = AT_QUERIES * HD * 2, K_BYTES = FRB_PAGE * HD * 2, V_BYTES = VD * FRB_PAGE * 2;
    constexpr uint32_t K_STEP = AP_STEP_PAGES * K_BYTES;                       // a step's keys of one map
    constexpr uint32_t STAGE_BYTES = 2 * K_STEP + AP_STEP_PAGES * V_BYTES;
    constexpr uint32_t SP_COL0 = 0, O_COL0 = 2 * AP_STEP_KEYS, TMEM_COLS = 512;

    let_next_kernel_start();
    const int tile = gridDim.x - 1 - blockIdx.x, head = blockIdx.y;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int group = p.heads / p.v_heads, vh = head / group;
    const int b = p.tile_seq[tile], q0 = p.tile_q0[tile];
    const int q_len = p.seq_q_len[b], start = p.seq_start[b], tok0 = p.cu_q_len[b] + q0;
    const int* table = p.page_table + (size_t)p.seq_slot[b] * p.max_pages;
    const int last_key = start + min(q0 + AT_QUERIES - 1, q_len - 1);
    const int first_page = first_visible_key(start + q0, p.window, 0) / FRB_PAGE;
    const int kept = kept_runs(p.keep_first, FRB_PAGE, first_page);
    const int num_pages = kept + last_key / FRB_PAGE - first_page + 1;
    const int num_steps = (num_pages + AP_STEP_PAGES - 1) / AP_STEP_PAGES;

    uint8_t* base = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    uint8_t* q_tiles = base;                                   // two maps x [128 x 64]
    uint8_t* stage0 = base + 2 * Q_BYTES;                      // per stage: K of map 1, K of map 2 ([128 keys x 64] each), V^T ([VD x 64] per page)

    if (threadIdx.x == 0) {
        bar_init(&q_full, 1);
        for (int s = 0; s < AP_STAGES; ++s) { bar_init(&kv_full[s], 1); bar_init(&kv_empty[s], 1); }
        for (int m = 0; m < 2; ++m) {
            bar_init(&s_full[m], 1);
            for (int h = 0; h < AP_STEP_PAGES; ++h) bar_init(&p_full[m][h], 4);
        }
        failed_flag = 0;
        bar_init_fence();
    }
    if (warp == 1) tmem_alloc(&tmem_slot, TMEM_COLS);
    fence_before_sync();
    __syncthreads();
    fence_after_sync();
    const uint32_t tmem = tmem_slot;
    wait_for_previous_kernel();

    if (warp == 0) {
        if (lane == 0) {
            bar_expect(&q_full, 2 * Q_BYTES);
            for (int m = 0; m < 2; ++m)
                load_2d(q_tiles + m * Q_BYTES, &map_q, ((vh * 2 + m) * group + head - vh * group) * HD, tok0, &q_full);
            for (int j = 0; j < num_steps; ++j) {
                const int s = j % AP_STAGES;
                if (!bar_wait(&kv_empty[s], ((j / AP_STAGES) & 1) ^ 1, failed)) { atomicExch(p.status, 31); break; }
                const int pages = min(AP_STEP_PAGES, num_pages - AP_STEP_PAGES * j);
                uint8_t* dst = stage0 + (size_t)s * STAGE_BYTES;
                bar_expect(&kv_full[s], pages * (2 * K_BYTES + V_BYTES));
                for (int h = 0; h < pages; ++h) {
                    const int page = table[run_at(AP_STEP_PAGES * j + h, kept, first_page)];
                    for (int m = 0; m < 2; ++m)
                        load_2d(dst + m * K_STEP + h * K_BYTES, &map_k, 0, ((page * p.v_heads + vh) * 2 + m) * FRB_PAGE, &kv_full[s]);
                    load_2d(dst + 2 * K_STEP + h * V_BYTES, &map_v, 0, (page * p.v_heads + vh) * VD, &kv_full[s]);
                }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t idesc_o = instr_desc_bf16(AT_QUERIES, VD);
            bool ok = bar_wait(&q_full, 0, failed);
            if (!ok) atomicExch(p.status, 32);
            auto issue_scores = [&](int m, int j) -> bool {
                const int s = j % AP_STAGES;
                if (!bar_wait(&kv_full[s], (j / AP_STAGES) & 1, failed)) { atomicExch(p.status, 33); return false; }
                fence_after_sync();
                const int pages = min(AP_STEP_PAGES, num_pages - AP_STEP_PAGES * j);
                const uint32_t idesc_s = instr_desc_bf16(AT_QUERIES, pages * FRB_PAGE);
                const uint64_t q_desc = tile_desc(smem_addr(q_tiles + m * Q_BYTES));
                const uint64_t k_desc = tile_desc(smem_addr(stage0 + (size_t)s * STAGE_BYTES + m * K_STEP));
#pragma unroll
                for (int k = 0; k < HD / 16; ++k)
                    mma_ss(tmem + SP_COL0 + AP_STEP_KEYS * m, q_desc + 2 * k, k_desc + 2 * k, idesc_s, k != 0);
                mma_commit(&s_full[m]);
                return true;
            };
            if (ok) ok = issue_scores(0, 0) && issue_scores(1, 0);
            for (int j = 0; j < num_steps && ok; ++j) {
                const int s = j % AP_STAGES;
                const int pages = min(AP_STEP_PAGES, num_pages - AP_STEP_PAGES * j);
                const uint64_t v_desc = tile_desc(smem_addr(stage0 + (size_t)s * STAGE_BYTES + 2 * K_STEP));
                for (int m = 0; m < 2 && ok; ++m) {
                    for (int h = 0; h < pages && ok; ++h) {
                        if (!bar_wait(&p_full[m][h], j & 1, failed)) { atomicExch(p.status, 35); ok = false; break; }
                        fence_after_sync();
#pragma unroll
                        for (int k = 0; k < 4; ++k)            // 16 keys per MMA: 8 columns of packed P, 32 bytes of a V^T row
                            mma_ts(tmem + O_COL0 + 128 * m, tmem + SP_COL0 + AP_STEP_KEYS * m + 64 * h + 8 * k,
                                   v_desc + ((h * V_BYTES + k * 32) >> 4), idesc_o, (j | h | k) != 0);
                    }
                    if (!ok) break;
                    if (m == 1) mma_commit(&kv_empty[s]);      // every product of the step has been issued: its stage, once they end
                    if (j + 1 < num_steps) ok = issue_scores(m, j + 1);
                }
            }
        }
    } else {
        const int quarter = warp & 3, m = (warp - 2) >> 2;
        const int row = quarter * 32 + lane;                   // the query row of this thread = its lane of tensor memory
        const uint32_t lane_base = tmem + ((uint32_t)(quarter * 32) << 16);
        const uint32_t mine = lane_base + SP_COL0 + AP_STEP_KEYS * m, o_mine = lane_base + O_COL0 + 128 * m;
        const bool valid = q0 + row < q_len;
        const int hi = valid ? start + q0 + row : -1;
        const int lo = valid ? first_visible_key(hi, p.window, 0) : 0;
        const float scale2 = CAPPED ? 1.f : p.scale2;
        float m_used = -INFINITY, l_sum = 0.f;
        bool ok = true;
        // whether every key of a page is visible to every row of the warp: most pages are, and need no comparisons
        auto open_page = [&](int key0) {
            return __all_sync(0xffffffffu, valid && key0 + FRB_PAGE - 1 <= hi && (key0 >= lo || key0 + FRB_PAGE <= p.keep_first));
        };
        for (int j = 0; j < num_steps; ++j) {
            // a wait that gives up does not end the loop: the block's later waits then return at once
            if (!bar_wait(&s_full[m], j & 1, failed)) { if (ok && lane == 0) atomicExch(p.status, 36); ok = false; }
            fence_after_sync();
            const int pages = min(AP_STEP_PAGES, num_pages - AP_STEP_PAGES * j);
            // the step's largest visible score, before its cap (which keeps the order)
            float step_max = -INFINITY;
#pragma unroll 1
            for (int h = 0; h < pages; ++h) {
                const int key0 = run_at(AP_STEP_PAGES * j + h, kept, first_page) * FRB_PAGE;
                uint32_t raw[FRB_PAGE / 16][16];
#pragma unroll
                for (int c = 0; c < FRB_PAGE / 16; ++c) tmem_ld16(mine + 64 * h + 16 * c, raw[c]);
                tmem_wait_ld();
                if (open_page(key0)) {
                    float top[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
                    for (int c = 0; c < FRB_PAGE / 16; ++c)
#pragma unroll
                        for (int i = 0; i < 16; i += 2)
                            top[(i >> 1) & 3] = max3(top[(i >> 1) & 3], __uint_as_float(raw[c][i]), __uint_as_float(raw[c][i + 1]));
                    step_max = fmaxf(step_max, fmaxf(fmaxf(top[0], top[1]), fmaxf(top[2], top[3])));
                } else {
#pragma unroll
                    for (int c = 0; c < FRB_PAGE / 16; ++c)
#pragma unroll
                        for (int i = 0; i < 16; ++i)
                            if (key_visible(key0 + 16 * c + i, lo, hi, p.keep_first)) step_max = fmaxf(step_max, __uint_as_float(raw[c][i]));
                }
            }
            if (step_max > -INFINITY) step_max = CAPPED ? capped_score2(step_max, p.cap_scale, p.cap2) : step_max * scale2;  // positive scale
            float corr = 1.f;
            const bool raise = step_max > m_used + AT_RAISE;   // also true on the first step with a visible key
            if (raise) { corr = exp2f(m_used - step_max); m_used = step_max; }
            if (j > 0 && __any_sync(0xffffffffu, raise)) {     // rare: O must follow the new maximum
#pragma unroll 1
                for (int c = 0; c < VD / 16; ++c) {
                    uint32_t o[16];
                    tmem_ld16(o_mine + 16 * c, o);
                    tmem_wait_ld();
#pragma unroll
                    for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * corr);
                    tmem_st16(o_mine + 16 * c, o);
                }
            }
            l_sum *= corr;
            const float m_sub = m_used == -INFINITY ? 0.f : m_used;
            const uint64_t scale_pair = pair_of(scale2, scale2), shift_pair = pair_of(-m_sub, -m_sub);
#pragma unroll 1
            for (int h = 0; h < pages; ++h) {
                const int key0 = run_at(AP_STEP_PAGES * j + h, kept, first_page) * FRB_PAGE;
                uint32_t raw[FRB_PAGE / 16][16];
#pragma unroll
                for (int c = 0; c < FRB_PAGE / 16; ++c) tmem_ld16(mine + 64 * h + 16 * c, raw[c]);
                tmem_wait_ld();
                if (CAPPED) cap_scores(raw, p.cap_scale, p.cap2);
                if (!open_page(key0)) {
#pragma unroll
                    for (int c = 0; c < FRB_PAGE / 16; ++c)
#pragma unroll
                        for (int i = 0; i < 16; ++i)
                            if (!key_visible(key0 + 16 * c + i, lo, hi, p.keep_first)) raw[c][i] = 0xff800000u;      // minus infinity
                }
                uint64_t sums[4] = {0ull, 0ull, 0ull, 0ull};
                uint32_t packed[FRB_PAGE / 32][16];
#pragma unroll
                for (int c = 0; c < FRB_PAGE / 16; ++c)
#pragma unroll
                    for (int i = 0; i < 16; i += 2) {
                        float x0, x1;
                        halves_of(fma_pairs(pair_of(__uint_as_float(raw[c][i]), __uint_as_float(raw[c][i + 1])), scale_pair, shift_pair), x0, x1);
                        const float a = exp2_fast(x0), bb = exp2_fast(x1);
                        sums[(i >> 1) & 3] = add_pairs(sums[(i >> 1) & 3], pair_of(a, bb));
                        packed[c >> 1][(c & 1) * 8 + (i >> 1)] = pack_bf16x2(a, bb);
                    }
                float sum_even, sum_odd;
                halves_of(add_pairs(add_pairs(sums[0], sums[1]), add_pairs(sums[2], sums[3])), sum_even, sum_odd);
                l_sum += sum_even + sum_odd;
#pragma unroll
                for (int c = 0; c < FRB_PAGE / 32; ++c) tmem_st16(mine + 64 * h + 16 * c, packed[c]);
                tmem_wait_st();
                fence_before_sync();
                __syncwarp();
                if (lane == 0) bar_arrive(&p_full[m][h]);
            }
        }
        {
            // a wait names a phase by its parity only: the step before the last one first
            const int last = num_steps - 1;
            if (last > 0 && !bar_wait(&kv_empty[(last - 1) % AP_STAGES], ((last - 1) / AP_STAGES) & 1, failed)) { if (ok && lane == 0) atomicExch(p.status, 39); ok = false; }
            if (!bar_wait(&kv_empty[last % AP_STAGES], (last / AP_STAGES) & 1, failed)) { if (ok && lane == 0) atomicExch(p.status, 39); ok = false; }
            fence_after_sync();
        }
        // Every MMA has ended and the stages are free: the two threads of a row exchange their maps' factors, and then what
        // their halves of the difference sum to.
        float* told = reinterpret_cast<float*>(stage0);        // [2 maps][128 rows], then [2 halves][128 rows]
        told[m * AT_QUERIES + row] = l_sum > 0.f ? 1.0f / l_sum : 0.f;
        asm volatile("bar.sync 1, %0;" ::"n"(AP_SOFTMAX_THREADS) : "memory");
        const float w1 = told[row], w2 = -*p.lam * told[AT_QUERIES + row];
        constexpr int MINE = VD / 2;                           // value entries of this thread: [MINE m, MINE m + MINE)
        float y[MINE], ss = 0.f;
#pragma unroll
        for (int c = 0; c < MINE / 16; ++c) {
            uint32_t o1[16], o2[16];
            tmem_ld16(lane_base + O_COL0 + MINE * m + 16 * c, o1);
            tmem_ld16(lane_base + O_COL0 + 128 + MINE * m + 16 * c, o2);
            tmem_wait_ld();
#pragma unroll
            for (int i = 0; i < 16; ++i) {
                const float o = fmaf(__uint_as_float(o2[i]), w2, __uint_as_float(o1[i]) * w1);
                y[16 * c + i] = o;
                ss = fmaf(o, o, ss);
            }
        }
        told[(2 + m) * AT_QUERIES + row] = ss;
        asm volatile("bar.sync 1, %0;" ::"n"(AP_SOFTMAX_THREADS) : "memory");
        const float mean = (told[2 * AT_QUERIES + row] + told[3 * AT_QUERIES + row]) / (float)VD;
        const float norm = p.factor / sqrtf(mean + p.eps);
        if (ok && !*failed && valid) {
            uint4* dst = reinterpret_cast<uint4*>(p.out + ((size_t)(tok0 + row) * p.heads + head) * VD + MINE * m);
#pragma unroll
            for (int c = 0; c < MINE / 8; ++c) {
                uint4 v;
                v.x = pack_bf16x2(y[8 * c] * norm, y[8 * c + 1] * norm);
                v.y = pack_bf16x2(y[8 * c + 2] * norm, y[8 * c + 3] * norm);
                v.z = pack_bf16x2(y[8 * c + 4] * norm, y[8 * c + 5] * norm);
                v.w = pack_bf16x2(y[8 * c + 6] * norm, y[8 * c + 7] * norm);
                dst[c] = v;
            }
        }
    }
    fence_before_sync();
    __syncthreads();
    if (failed_flag && warp == 0 && lane == 0) {
        // copies may still be on their way into this block's shared memory: give them a bounded time to land
        int zero = 0;
        bar_wait(&q_full, 0, &zero);
        for (int s = 0; s < AP_STAGES; ++s) { zero = 0; bar_wait(&kv_full[s], 0, &zero); }
    }
    __syncthreads();
    if (warp == 1) tmem_free(tmem, TMEM_COLS);
}

// q bf16 [num_tokens, v_heads, 2, group, hd]; k_pages [pages, v_heads, 2, 64, hd]; v_pages [pages, v_heads, vd, 64]; tiles of 128
// queries; out bf16 [num_tokens, heads, vd].  lam: one float32 on the device.  status: one int on the device, zero before the call.
FRB_API int frb_attention_pair_tc(const void* q, int num_tokens, const void* k_pages, const void* v_pages, int num_pages,
                                  const int* page_table, int max_pages, const int* tile_seq, const int* tile_q0, int num_tiles,
                                  const int* seq_slot, const int* seq_start, const int* seq_q_len, const int* cu_q_len, void* out,
                                  int heads, int v_heads, int head_dim, int v_dim, float scale, int window, int keep_first, float softcap,
                                  const float* lam, float eps, float factor, int* status, cudaStream_t stream) {
    if (num_tiles == 0) return 0;
    FRB_CHECK_ARG(head_dim == 64 && (v_dim == 64 || v_dim == 128), "attention of two maps: head_dim %d with value heads of %d is not built",
                  head_dim, v_dim);
    FRB_CHECK_ARG(scale > 0.f && keep_first >= 0, "attention of two maps: a softmax scale of %g", (double)scale);
    FRB_CHECK_ARG(v_heads > 0 && heads % v_heads == 0 && heads <= 65535, "attention of two maps: %d heads over %d value heads", heads, v_heads);
    CUtensorMap map_q, map_k, map_v;
    FRB_CHECK_ARG(map_rows_of_64(&map_q, q, num_tokens, (uint64_t)2 * heads * head_dim, AT_QUERIES) &&
                  map_rows_of_64(&map_k, k_pages, (uint64_t)num_pages * 2 * v_heads * FRB_PAGE, head_dim, FRB_PAGE) &&
                  map_rows_of_64(&map_v, v_pages, (uint64_t)num_pages * v_heads * v_dim, FRB_PAGE, v_dim),
                  "attention of two maps: cuTensorMapEncodeTiled failed or is not available");
    AttnPairParams p;
    p.page_table = page_table; p.tile_seq = tile_seq; p.tile_q0 = tile_q0; p.seq_slot = seq_slot; p.seq_start = seq_start;
    p.seq_q_len = seq_q_len; p.cu_q_len = cu_q_len; p.out = (bf16*)out; p.lam = lam; p.status = status;
    p.scale2 = scale * 1.4426950408889634f;
    p.cap_scale = softcap > 0.f ? scale / softcap : 0.f; p.cap2 = softcap > 0.f ? softcap * 1.4426950408889634f : 0.f;
    p.eps = eps; p.factor = factor; p.window = window; p.keep_first = window > 0 ? keep_first : 0; p.max_pages = max_pages;
    p.heads = heads; p.v_heads = v_heads;
    const size_t smem = (size_t)2 * AT_QUERIES * head_dim * 2 + (size_t)AP_STAGES * AP_STEP_PAGES * FRB_PAGE * (2 * head_dim + v_dim) * 2 + 1024;
    dim3 grid(num_tiles, heads);
#define FRB_LAUNCH_PAIR(VD, CAPPED)                                                                              \
    do {                                                                                                         \
        auto kernel = attention_pair_tc_kernel<64, VD, CAPPED>;                                                  \
        cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                    \
        launch_dependent(kernel, grid, dim3(AP_THREADS), smem, stream, map_q, map_k, map_v, p);                  \
    } while (0)
    if (v_dim == 128) { if (softcap > 0.f) FRB_LAUNCH_PAIR(128, true); else FRB_LAUNCH_PAIR(128, false); }
    else { if (softcap > 0.f) FRB_LAUNCH_PAIR(64, true); else FRB_LAUNCH_PAIR(64, false); }
#undef FRB_LAUNCH_PAIR
    FRB_RETURN_LAUNCH("attention_pair_tc");
}
