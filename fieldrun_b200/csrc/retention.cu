// Retention: linear attention with one fixed decay per head, over a float32 state S [dim, vdim] per sequence and head.
//
//   S_t = decay S_(t-1) + (k_scale k_t) v_t^T,    o_t = S_t^T q_t                          the read-out sees the token's own write
//   out = o / sqrt(mean(o^2) + eps) * silu(g)                                              over the head's vdim values, no weight
//
// The state of a slot exists twice, [slot][2][copy_floats]: a step that begins at position p reads copy (p & 1) and writes copy
// ((p + n) & 1) after its n tokens, so a step of one token never writes what it reads.  Every element of the state is read and
// written by one thread.  A decay is kept less one and applied as S + (decay - 1) S: rounded to float32, a decay itself loses its
// distance from one, by the same amount at every token.
#include "common.cuh"

#define RET_TOKENS 8           // tokens whose rows are asked for together
#define RET_CHUNK 64           // tokens of a chunk of the tensor-core kernel; the decay tables reach this far

struct RetentionParams {
    const float* proj;       // [T, proj_stride]: q at q_off (heads * dim), k at k_off, v at v_off (heads * vdim), gate at g_off
    const float* decays;     // [heads][2][RET_CHUNK + 1]: decay^n, then decay^n - 1
    const int* seq_slot;     // [B]
    const int* seq_start;    // [B]
    const int* cu_q_len;     // [B + 1]
    float* state;
    long long copy_floats, state_offset;
    void* out;               // [T, heads * vdim]
    float* raw;              // null, or [T, heads * vdim]: o before norm and gate (a head's value columns are cut over blocks)
    int proj_stride, q_off, k_off, v_off, g_off, heads, dim, vdim, parts, npad;
    float k_scale, eps;
};

__device__ __forceinline__ void ret_copy_async4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void ret_copies_wait() { asm volatile("cp.async.wait_all;" ::: "memory"); }

// Norm and gate of one head's output by one warp; o(d) gives the output's entry d.
template <typename OutT, typename Entry>
__device__ __forceinline__ void ret_finish(Entry o, const float* gate, OutT* out, int vdim, float eps, int lane) {
    float ss = 0.f;
    for (int d = lane; d < vdim; d += 32) { const float v = o(d); ss += v * v; }
    const float rinv = 1.0f / sqrtf(warp_sum(ss) / (float)vdim + eps);
    for (int d = lane; d < vdim; d += 32) {
        const float z = gate[d];
        out[d] = from_f32<OutT>(o(d) * rinv * (z / (1.0f + expf(-z))));
    }
}

// The recurrence token by token.  A block takes (sequence, head, slice of 32 VP value columns); warp `part` keeps NREG rows of
// the state for each of its lane's VP columns (v = lane + 32 j).  Tokens go eight at a time: while the eight steps of one buffer
// run (without a barrier) the rows of the next eight are on their way into the other.  The warps' shares of o are added in
// warp order.
template <int NREG, int VP, typename OutT>
__global__ void __launch_bounds__(512) retention_token_kernel(RetentionParams p) {
    extern __shared__ __align__(16) float sm[];
    after_previous_kernel();
    constexpr int COLS = 32 * VP;
    const int dim = p.dim, npad = p.npad, parts = p.parts, vdim = p.vdim;
    const int buffer_floats = RET_TOKENS * (2 * npad + COLS);
    float* s_o = sm + 2 * buffer_floats;               // [RET_TOKENS][parts][COLS]
    const int b = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * COLS;
    const int lane = threadIdx.x & 31, part = threadIdx.x >> 5;
    const int row0 = p.cu_q_len[b], n_tok = p.cu_q_len[b + 1] - row0;
    const int start = p.seq_start[b], slot = p.seq_slot[b];
    const int n0 = part * NREG;
    float* state = p.state + (size_t)slot * 2 * p.copy_floats + p.state_offset + (size_t)h * dim * vdim;
    const float* s_in = state + (start & 1) * p.copy_floats;
    float* s_out = state + ((start + n_tok) & 1) * p.copy_floats;
    float S[NREG][VP];
#pragma unroll
    for (int i = 0; i < NREG; ++i)
#pragma unroll
        for (int j = 0; j < VP; ++j) {
            const int v = v0 + lane + 32 * j;
            S[i][j] = (v < vdim && n0 + i < dim) ? s_in[(size_t)(n0 + i) * vdim + v] : 0.f;
        }
    const float less = p.decays[((size_t)h * 2 + 1) * (RET_CHUNK + 1) + 1];
    for (int i = threadIdx.x; i < 2 * buffer_floats; i += blockDim.x) sm[i] = 0.f;      // the padding stays zero
    __syncthreads();
    const int chunks = (n_tok + RET_TOKENS - 1) / RET_TOKENS;

    auto stage = [&](int n) {
        float* s_q = sm + (n & 1) * buffer_floats;
        float* s_k = s_q + RET_TOKENS * npad;
        float* s_v = s_k + RET_TOKENS * npad;
        const int t0 = n * RET_TOKENS, count = min(RET_TOKENS, n_tok - t0);
        for (int t = part; t < count; t += parts) {
            const float* row = p.proj + (size_t)(row0 + t0 + t) * p.proj_stride;
            for (int d = lane; d < dim; d += 32) {
                ret_copy_async4(s_q + t * npad + d, row + p.q_off + h * dim + d);
                ret_copy_async4(s_k + t * npad + d, row + p.k_off + h * dim + d);
            }
            for (int d = lane; d < COLS && v0 + d < vdim; d += 32) ret_copy_async4(s_v + t * COLS + d, row + p.v_off + h * vdim + v0 + d);
        }
    };

    stage(0);
    for (int n = 0; n < chunks; ++n) {
        const int t0 = n * RET_TOKENS, count = min(RET_TOKENS, n_tok - t0);
        ret_copies_wait();
        __syncthreads();                               // chunk n lies in its buffer; nobody reads the other one any more
        if (n + 1 < chunks) stage(n + 1);
        const float* s_q = sm + (n & 1) * buffer_floats;
        const float* s_k = s_q + RET_TOKENS * npad;
        const float* s_v = s_k + RET_TOKENS * npad;
#pragma unroll
        for (int t = 0; t < RET_TOKENS; ++t) {
            if (t < count) {
                float vs[VP], o[VP];
#pragma unroll
                for (int j = 0; j < VP; ++j) { vs[j] = p.k_scale * s_v[t * COLS + lane + 32 * j]; o[j] = 0.f; }
#pragma unroll
                for (int i = 0; i < NREG; i += 4) {
                    const float4 k4 = *reinterpret_cast<const float4*>(s_k + t * npad + n0 + i);
                    const float4 q4 = *reinterpret_cast<const float4*>(s_q + t * npad + n0 + i);
                    const float kk[4] = {k4.x, k4.y, k4.z, k4.w}, qq[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
                    for (int u = 0; u < 4; ++u)
#pragma unroll
                        for (int j = 0; j < VP; ++j) {
                            S[i + u][j] = fmaf(kk[u], vs[j], fmaf(less, S[i + u][j], S[i + u][j]));
                            o[j] = fmaf(S[i + u][j], qq[u], o[j]);
                        }
                }
#pragma unroll
                for (int j = 0; j < VP; ++j) s_o[(t * parts + part) * COLS + lane + 32 * j] = o[j];
            }
        }
        __syncthreads();
        for (int t = part; t < count; t += parts) {
            const size_t row = (size_t)(row0 + t0 + t);
            float* o = s_o + t * parts * COLS;
            for (int d = lane; d < COLS; d += 32) {
                float sum = o[d];
                for (int q = 1; q < parts; ++q) sum += o[q * COLS + d];
                o[d] = sum;
                if (p.raw && v0 + d < vdim) p.raw[(row * p.heads + h) * vdim + v0 + d] = sum;
            }
            __syncwarp();
            if (!p.raw)
                ret_finish<OutT>([&](int d) { return o[d]; }, p.proj + row * p.proj_stride + p.g_off + h * vdim,
                                 (OutT*)p.out + (row * p.heads + h) * vdim, vdim, p.eps, lane);
        }
    }
#pragma unroll
    for (int i = 0; i < NREG; ++i)
#pragma unroll
        for (int j = 0; j < VP; ++j) {
            const int v = v0 + lane + 32 * j;
            if (v < vdim && n0 + i < dim) s_out[(size_t)(n0 + i) * vdim + v] = S[i][j];
        }
}

// Norms and gates the outputs that blocks of a part of a head left in `raw`: a warp per (token, head).
template <typename OutT>
__global__ void __launch_bounds__(128) retention_output_kernel(RetentionParams p, int num_rows) {
    after_previous_kernel();
    const int lane = threadIdx.x & 31, item = blockIdx.x * 4 + (threadIdx.x >> 5);
    if (item >= num_rows * p.heads) return;
    const size_t row = item / p.heads;
    const int h = item - (int)row * p.heads;
    const float* o = p.raw + (row * p.heads + h) * p.vdim;
    ret_finish<OutT>([&](int d) { return o[d]; }, p.proj + row * p.proj_stride + p.g_off + h * p.vdim,
                     (OutT*)p.out + (row * p.heads + h) * p.vdim, p.vdim, p.eps, lane);
}

FRB_API int frb_retention(const float* proj, int proj_stride, int q_off, int k_off, int v_off, int g_off, const float* decays,
                          const int* seq_slot, const int* seq_start, const int* cu_q_len, float* state, long long copy_floats,
                          long long state_offset, void* out, int out_dtype, float* raw, int num_rows, int num_seqs, int heads, int dim,
                          int vdim, float k_scale, float eps, cudaStream_t stream) {
    if (num_seqs == 0) return 0;
    FRB_CHECK_ARG(heads >= 1 && heads <= 65535 && vdim >= 1, "retention: %d heads of %d x %d", heads, dim, vdim);
    FRB_CHECK_ARG(dim >= 1 && dim <= 1024, "retention: %d keys a head are outside 1..1024", dim);
    RetentionParams p;
    p.proj = proj; p.decays = decays; p.seq_slot = seq_slot; p.seq_start = seq_start; p.cu_q_len = cu_q_len; p.state = state;
    p.copy_floats = copy_floats; p.state_offset = state_offset; p.out = out; p.proj_stride = proj_stride; p.q_off = q_off;
    p.k_off = k_off; p.v_off = v_off; p.g_off = g_off; p.heads = heads; p.dim = dim; p.vdim = vdim; p.k_scale = k_scale; p.eps = eps;
    int nreg = 8;
    while ((dim + nreg - 1) / nreg > 16) nreg <<= 1;
    // value columns a lane: as many as the head has (in 32s) while a thread's share of the state stays within 64 registers
    int vp = vdim > 64 ? 4 : vdim > 32 ? 2 : 1;
    while (vp > 1 && nreg * vp > 64) vp >>= 1;
    const int cols = 32 * vp, slices = (vdim + cols - 1) / cols;
    FRB_CHECK_ARG(slices <= 65535, "retention: %d slices exceed the grid", slices);
    FRB_CHECK_ARG(slices == 1 || raw, "retention: heads of %d x %d go over %d blocks each, which needs the float32 buffer for their outputs",
                  dim, vdim, slices);
    p.raw = slices > 1 ? raw : nullptr;
    p.parts = (dim + nreg - 1) / nreg;
    p.npad = p.parts * nreg;
    const size_t smem = (2 * (size_t)RET_TOKENS * (2 * p.npad + cols) + (size_t)RET_TOKENS * p.parts * cols) * sizeof(float);
    FRB_CHECK_ARG(smem <= 200 * 1024, "retention: heads of %d x %d need %zu bytes of shared memory", dim, vdim, smem);
    const dim3 grid(num_seqs, heads, slices), block(32 * p.parts);
#define FRB_RET(NREG, VP)                                                                                              \
    do {                                                                                                               \
        auto kernel = retention_token_kernel<NREG, VP, OutT>;                                                          \
        if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);    \
        launch_dependent(kernel, grid, block, smem, stream, p);                                                        \
    } while (0)
    FRB_DISPATCH_DTYPE(out_dtype, OutT, {
        if (nreg == 8) { if (vp == 4) FRB_RET(8, 4); else if (vp == 2) FRB_RET(8, 2); else FRB_RET(8, 1); }
        else if (nreg == 16) { if (vp == 4) FRB_RET(16, 4); else if (vp == 2) FRB_RET(16, 2); else FRB_RET(16, 1); }
        else if (nreg == 32) { if (vp == 2) FRB_RET(32, 2); else FRB_RET(32, 1); }
        else FRB_RET(64, 1);
        if (p.raw)
            launch_dependent(retention_output_kernel<OutT>, dim3((num_rows * heads + 3) / 4), dim3(128), 0, stream, p, num_rows);
    });
#undef FRB_RET
    FRB_RETURN_LAUNCH("retention");
}
