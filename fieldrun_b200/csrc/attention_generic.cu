// Attention over the paged cache, any head size up to 256 and any group size, float32 arithmetic.
// It is the whole attention of the float32 path and the fallback of the bfloat16 path for shapes that
// the tensor-core kernels refuse.
//
// Per query head h with kv = h / (nh / nkv): s_j = (q . K_j) * scale for the keys the query may see
// (j <= its position, and j > position - window when a window is set), p = exp(s - max) / sum,
// out = sum_j p_j V_j  (src/minimax.rs:270-281).  Keys that are hidden get weight 0 exactly, which is what
// the reference's -1e30 amounts to after the exponential.
// Two things the reference's model does not have are arguments here: a value head of another size than the
// key head (v_dim), and a bias on the score that grows with the distance, s_j -= slope[h] * (i - j) for the query
// at position i (a slope per query head; null: none).  Three more, each off unless given: `chunk` (the query at i
// sees only keys of its own chunk, floor(j / chunk) == floor(i / chunk), chunks counted from position 0), `sinks`
// (a number per query head whose exponential joins the softmax's denominator, with no key and no value: it is not
// scaled and counts once), `gate` (the head's output is multiplied by sigmoid(gate[t, h])) and `softcap` (the scaled
// score s of every key becomes softcap * tanh(s / softcap) before anything else is done with it).  `keep_first`: beside the
// window the query sees the sequence's first tokens.  Key heads in runs of num_kv_heads / num_v_heads share a value head (two
// maps over one set of values); the output may be float32 whatever the operands are.
#include "common.cuh"

struct AttnParams {
    const void* q;            // [T, nh, hd]
    const void* k_pages;      // [pages, nkv, PAGE, hd]
    const void* v_pages;      // [pages, nkv, vd, PAGE]: values lie transposed within a page
    const float* slopes;      // [nh] or null
    const float* sinks;       // [nh] or null
    const float* gate;        // [T, gate_stride] or null: head h of token t at t * gate_stride + h
    int chunk, gate_stride;   // chunk 0: no chunks
    const int* page_table;    // [slots, max_pages]
    const int* tok_pos;       // [T]
    const int* tok_slot;      // [T]
    void* out;                // [T, nh * vd]
    int out_f32;              // the output is float32 whatever T is
    int keep_first, v_heads;
    float scale;
    float softcap;            // > 0: the scaled score s becomes softcap * tanh(s / softcap); 0: none
    int window;               // 0: every earlier key
    int max_pages, num_heads, num_kv_heads, head_dim, v_dim;
};

#define KEY_BLOCK 32

// grid (token, kv head); one warp per query head of the group, warps share the staged K/V block.
template <typename T>
__global__ void attention_generic_kernel(AttnParams p) {
    extern __shared__ float sm[];
    const int hd = p.head_dim, vd = p.v_dim;
    float* k_tile = sm;                                  // [KEY_BLOCK][hd + 1]
    float* v_tile = k_tile + KEY_BLOCK * (hd + 1);       // [KEY_BLOCK][vd]
    float* q_rows = v_tile + KEY_BLOCK * vd;             // [warps][hd]
    const int t = blockIdx.x, g = blockIdx.y;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
    const int group = p.num_heads / p.num_kv_heads;
    const int pos = p.tok_pos[t];
    const int hi = pos;
    int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
    if (p.chunk > 0) lo = max(lo, pos / p.chunk * p.chunk);
    const int* table = p.page_table + (size_t)p.tok_slot[t] * p.max_pages;
    const T* q = (const T*)p.q;
    const T* k_pages = (const T*)p.k_pages;
    const T* v_pages = (const T*)p.v_pages;
    const int vg = g / (p.num_kv_heads / p.v_heads);
    const int first_block = lo / KEY_BLOCK, kept = kept_runs(p.keep_first, KEY_BLOCK, first_block);
    const int blocks = kept + hi / KEY_BLOCK - first_block + 1;

    for (int hbase = 0; hbase < group; hbase += nwarps) {
        const int hl = hbase + warp;
        const bool active = hl < group;
        const int head = g * group + hl;
        if (active)
            for (int d = lane; d < hd; d += 32) q_rows[warp * hd + d] = to_f32<T>(q[((size_t)t * p.num_heads + head) * hd + d]);
        const float slope = (active && p.slopes) ? p.slopes[head] : 0.f;
        float m = -INFINITY, l = 0.f;
        float acc[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) acc[i] = 0.f;

        for (int n = 0; n < blocks; ++n) {
            const int j0 = run_at(n, kept, first_block) * KEY_BLOCK;
            __syncthreads();
            const int page = table[j0 / FRB_PAGE];
            const size_t head_base = ((size_t)page * p.num_kv_heads + g) * FRB_PAGE * hd;
            const size_t value_base = ((size_t)page * p.v_heads + vg) * FRB_PAGE * vd;
            const int in_page = j0 % FRB_PAGE;
            for (int i = threadIdx.x; i < KEY_BLOCK * hd; i += blockDim.x) {
                const int r = i / hd, d = i - r * hd;
                const bool valid = key_visible(j0 + r, lo, hi, p.keep_first);
                k_tile[r * (hd + 1) + d] = valid ? to_f32<T>(k_pages[head_base + (size_t)(in_page + r) * hd + d]) : 0.f;
            }
            for (int i = threadIdx.x; i < KEY_BLOCK * vd; i += blockDim.x) {
                const int d = i / KEY_BLOCK, r = i - d * KEY_BLOCK;          // keys of one dim are neighbours in memory
                const bool valid = key_visible(j0 + r, lo, hi, p.keep_first);
                v_tile[r * vd + d] = valid ? to_f32<T>(v_pages[value_base + (size_t)d * FRB_PAGE + in_page + r]) : 0.f;
            }
            __syncthreads();
            if (active) {
                const int j = j0 + lane;
                const bool valid = key_visible(j, lo, hi, p.keep_first);
                float s = 0.f;
                const float* qr = q_rows + warp * hd;
                const float* kr = k_tile + lane * (hd + 1);
                for (int d = 0; d < hd; ++d) s += qr[d] * kr[d];
                s *= p.scale;
                if (p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
                s = valid ? s - slope * (float)(pos - j) : -INFINITY;
                const float m_new = fmaxf(m, warp_max(s));
                const float corr = expf(m - m_new);
                const float pj = valid ? expf(s - m_new) : 0.f;
                l = l * corr + warp_sum(pj);
#pragma unroll
                for (int i = 0; i < 8; ++i) acc[i] *= corr;
                for (int kk = 0; kk < KEY_BLOCK; ++kk) {
                    const float pk = __shfl_sync(0xffffffffu, pj, kk);
#pragma unroll
                    for (int i = 0; i < 8; ++i) {
                        const int d = lane + 32 * i;
                        if (d < vd) acc[i] += pk * v_tile[kk * vd + d];
                    }
                }
                m = m_new;
            }
        }
        if (active) {
            if (p.sinks) {
                const float sink = p.sinks[head];
                const float m_new = fmaxf(m, sink);
                const float corr = expf(m - m_new);
                l = l * corr + expf(sink - m_new);
#pragma unroll
                for (int i = 0; i < 8; ++i) acc[i] *= corr;
            }
            float inv = 1.0f / l;
            if (p.gate) inv *= 1.0f / (1.0f + expf(-p.gate[(size_t)t * p.gate_stride + head]));
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const int d = lane + 32 * i;
                const size_t at = ((size_t)t * p.num_heads + head) * vd + d;
                if (d < vd) {
                    if (p.out_f32) ((float*)p.out)[at] = acc[i] * inv;
                    else ((T*)p.out)[at] = from_f32<T>(acc[i] * inv);
                }
            }
        }
    }
}

FRB_API int frb_attention_generic(const void* q, const void* k_pages, const void* v_pages, int dtype,
                                  const int* page_table, int max_pages, const int* tok_pos, const int* tok_slot,
                                  void* out, int num_tokens, int num_heads, int num_kv_heads, int head_dim,
                                  float scale, int window, int v_dim, const float* slopes, int chunk, const float* sinks,
                                  const float* gate, int gate_stride, float softcap, int keep_first, int num_v_heads, int out_f32,
                                  cudaStream_t stream) {
    if (num_tokens == 0) return 0;
    if (num_v_heads <= 0) num_v_heads = num_kv_heads;
    FRB_CHECK_ARG(num_kv_heads % num_v_heads == 0, "attention: %d key heads over %d value heads", num_kv_heads, num_v_heads);
    FRB_CHECK_ARG(keep_first >= 0 && !(keep_first > 0 && chunk > 0), "attention: %d first tokens together with chunks", keep_first);
    if (v_dim <= 0) v_dim = head_dim;
    FRB_CHECK_ARG(v_dim <= 256, "attention: v_dim %d is outside 1..256", v_dim);
    FRB_CHECK_ARG(head_dim >= 1 && head_dim <= 256, "attention: head_dim %d is outside 1..256", head_dim);
    FRB_CHECK_ARG(num_kv_heads >= 1 && num_heads % num_kv_heads == 0, "attention: %d heads are not a multiple of %d kv heads",
                  num_heads, num_kv_heads);
    FRB_CHECK_ARG(num_kv_heads <= 65535, "attention: %d kv heads exceed the grid", num_kv_heads);
    AttnParams p;
    p.q = q; p.k_pages = k_pages; p.v_pages = v_pages; p.page_table = page_table; p.tok_pos = tok_pos;
    p.tok_slot = tok_slot; p.out = out; p.scale = scale; p.window = window; p.max_pages = max_pages;
    p.num_heads = num_heads; p.num_kv_heads = num_kv_heads; p.head_dim = head_dim; p.v_dim = v_dim; p.slopes = slopes;
    p.chunk = chunk; p.sinks = sinks; p.gate = gate; p.gate_stride = gate_stride; p.softcap = softcap;
    p.keep_first = window > 0 ? keep_first : 0; p.v_heads = num_v_heads; p.out_f32 = out_f32;
    const int group = num_heads / num_kv_heads;
    const int nwarps = group < 8 ? group : 8;
    const size_t smem = ((size_t)KEY_BLOCK * (head_dim + 1) + (size_t)KEY_BLOCK * v_dim + (size_t)nwarps * head_dim) * sizeof(float);
    dim3 grid(num_tokens, num_kv_heads);
    FRB_DISPATCH_DTYPE(dtype, T, {
        auto kernel = attention_generic_kernel<T>;
        if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        kernel<<<grid, 32 * nwarps, smem, stream>>>(p);
    });
    FRB_RETURN_LAUNCH("attention_generic");
}
