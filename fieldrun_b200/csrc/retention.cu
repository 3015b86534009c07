// Retention: linear attention with one fixed decay per head, over a float32 state S [dim, vdim] per sequence and head.
//
//   S_t = decay S_(t-1) + (k_scale k_t) v_t^T,    o_t = S_t^T q_t                          the read-out sees the token's own write
//   out = o / sqrt(mean(o^2) + eps) * silu(g)                                              over the head's vdim values, no weight
//
// The state of a slot exists twice, [slot][2][copy_floats]: a step that begins at position p reads copy (p & 1) and writes copy
// ((p + n) & 1) after its n tokens, so a step of one token never writes what it reads.  Every element of the state is read and
// written by one thread.  A decay is kept less one and applied as S + (decay - 1) S: rounded to float32, a decay itself loses its
// distance from one, by the same amount at every token.
//
// Two kernels.  The recurrence token by token, in float32, takes any sizes, single tokens and float32 models.  Prompts in
// bfloat16 go chunk by chunk on tensor cores (mma.sync): with i, j counted in a chunk of n tokens,
//     o_i = sum_{j <= i} decay^(i-j) (q_i . k_j) v_j + decay^(i+1) S^T q_i,      S <- decay^n S + sum_j decay^(n-1-j) k_j v_j^T
// (k_scale on every k).  q, k and v are bfloat16 there, as projections may be; everything else that enters a product, the
// decayed scores, the decayed values and the state, is float32 and goes in as the sum of three bfloat16 numbers (24 bits), so
// that the products are those of float32 operands; sums and the state are float32.
#include "common.cuh"

#define RET_TOKENS 8           // tokens whose rows are asked for together
#define RET_CHUNK 64           // tokens of a chunk of the tensor-core kernel; the decay tables reach this far

struct RetentionParams {
    const void* proj;        // [T, proj_stride], float32 (bfloat16 for the tensor-core kernel): q at q_off (heads * dim), k at k_off, v at v_off (heads * vdim), gate at g_off
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
template <typename OutT, typename GateT, typename Entry>
__device__ __forceinline__ void ret_finish(Entry o, const GateT* gate, OutT* out, int vdim, float eps, int lane) {
    float ss = 0.f;
    for (int d = lane; d < vdim; d += 32) { const float v = o(d); ss += v * v; }
    const float rinv = 1.0f / sqrtf(warp_sum(ss) / (float)vdim + eps);
    for (int d = lane; d < vdim; d += 32) {
        const float z = to_f32<GateT>(gate[d]);
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
    const float* proj = (const float*)p.proj;
    for (int i = threadIdx.x; i < 2 * buffer_floats; i += blockDim.x) sm[i] = 0.f;      // the padding stays zero
    __syncthreads();
    const int chunks = (n_tok + RET_TOKENS - 1) / RET_TOKENS;

    auto stage = [&](int n) {
        float* s_q = sm + (n & 1) * buffer_floats;
        float* s_k = s_q + RET_TOKENS * npad;
        float* s_v = s_k + RET_TOKENS * npad;
        const int t0 = n * RET_TOKENS, count = min(RET_TOKENS, n_tok - t0);
        for (int t = part; t < count; t += parts) {
            const float* row = proj + (size_t)(row0 + t0 + t) * p.proj_stride;
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
                ret_finish<OutT, float>([&](int d) { return o[d]; }, proj + row * p.proj_stride + p.g_off + h * vdim,
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
template <typename OutT, typename GateT>
__global__ void __launch_bounds__(128) retention_output_kernel(RetentionParams p, int num_rows) {
    after_previous_kernel();
    const int lane = threadIdx.x & 31, item = blockIdx.x * 4 + (threadIdx.x >> 5);
    if (item >= num_rows * p.heads) return;
    const size_t row = item / p.heads;
    const int h = item - (int)row * p.heads;
    const float* o = p.raw + (row * p.heads + h) * p.vdim;
    ret_finish<OutT, GateT>([&](int d) { return o[d]; }, (const GateT*)p.proj + row * p.proj_stride + p.g_off + h * p.vdim,
                     (OutT*)p.out + (row * p.heads + h) * p.vdim, p.vdim, p.eps, lane);
}

// ---------------------------------------------------------------------------------------------------- chunks on tensor cores

#define RET_PAD 8              // bfloat16 entries behind every row of a tile: eight rows of a matrix then lie in different banks

__device__ __forceinline__ void ret_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ret_matrices(uint32_t (&r)[4], const bf16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)) : "memory");
}
__device__ __forceinline__ void ret_matrices_turned(uint32_t (&r)[4], const bf16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)) : "memory");
}
__device__ __forceinline__ void ret_copy_async16(bf16* dst, const bf16* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
// two float32 numbers as three pairs of bfloat16 whose sums they are (to the last bit of a float32, or nearly)
__device__ __forceinline__ void ret_split(float x, float y, uint32_t (&part)[3]) {
#pragma unroll
    for (int s = 0; s < 3; ++s) {
        const __nv_bfloat162 v = __floats2bfloat162_rn(x, y);
        part[s] = *reinterpret_cast<const uint32_t*>(&v);
        x -= __low2float(v);
        y -= __high2float(v);
    }
}
__device__ __forceinline__ float ret_low(uint32_t v) { return __uint_as_float(v << 16); }
__device__ __forceinline__ float ret_high(uint32_t v) { return __uint_as_float(v & 0xffff0000u); }

// A block takes (sequence, head, slice of 16 W value columns), a warp 16 of those columns; DIM: the head's keys, padded with
// zeros.  A warp keeps its part of the state transposed, [16 value columns][DIM keys], as the accumulators of S^T += V^T K: the
// fragments are at the same time the left operand of o^T = S^T q^T.  The scores of a chunk are made by all warps together and
// pass through shared memory.  The next chunk's rows are on their way while a chunk runs.
template <int DIM, int W>
__global__ void __launch_bounds__(32 * W) retention_chunk_kernel(RetentionParams p) {
    extern __shared__ __align__(16) uint8_t raw_smem[];
    after_previous_kernel();
    constexpr int C = RET_CHUNK, VS = 16 * W;
    constexpr int K_ROW = DIM + RET_PAD, V_ROW = VS + RET_PAD, P_ROW = C + RET_PAD;
    constexpr int STAGE = C * (2 * K_ROW + V_ROW), P_PART = C * P_ROW;
    bf16* tiles = reinterpret_cast<bf16*>(raw_smem);            // two stages of q [C][K_ROW], k [C][K_ROW], v [C][V_ROW]
    bf16* s_p = tiles + 2 * STAGE;                              // three parts of the decayed scores [C][P_ROW]
    float* s_pow = reinterpret_cast<float*>(s_p + 3 * P_PART);  // [C + 1] decay^n
    float* s_w = s_pow + C + 1;                                 // [C] k_scale decay^(n-1-j), 0 for tokens that are not there
    const int b = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * VS;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
    const int m8 = lane >> 3, r8 = lane & 7;                    // the matrix and row that this lane names in an ldmatrix
    const int dim = p.dim, vdim = p.vdim;
    const int row0 = p.cu_q_len[b], n_tok = p.cu_q_len[b + 1] - row0;
    const int start = p.seq_start[b], slot = p.seq_slot[b];
    float* state = p.state + (size_t)slot * 2 * p.copy_floats + p.state_offset + (size_t)h * dim * vdim;
    const float* s_in = state + (start & 1) * p.copy_floats;
    float* s_out = state + ((start + n_tok) & 1) * p.copy_floats;
    const bf16* proj = (const bf16*)p.proj + (size_t)row0 * p.proj_stride;
    const int chunks = (n_tok + C - 1) / C;

    for (int i = threadIdx.x; i < STAGE; i += 32 * W) reinterpret_cast<uint32_t*>(tiles)[i] = 0u;       // the padding stays zero
    for (int i = threadIdx.x; i <= C; i += 32 * W) s_pow[i] = p.decays[(size_t)h * 2 * (C + 1) + i];
    __syncthreads();

    auto stage = [&](int n) {
        bf16* q = tiles + (n & 1) * STAGE;
        bf16* k = q + C * K_ROW;
        bf16* v = k + C * K_ROW;
        const int count = min(C, n_tok - n * C);
        const bf16* src = proj + (size_t)n * C * p.proj_stride;
        const int pieces = dim / 8, v_pieces = min(VS, vdim - v0) / 8;           // 16-byte pieces of a row
        for (int i = threadIdx.x; i < C * pieces; i += 32 * W) {
            const int r = i / pieces, d = (i - r * pieces) * 8;
            if (r < count) {
                ret_copy_async16(q + r * K_ROW + d, src + (size_t)r * p.proj_stride + p.q_off + h * dim + d);
                ret_copy_async16(k + r * K_ROW + d, src + (size_t)r * p.proj_stride + p.k_off + h * dim + d);
            } else {
                *reinterpret_cast<uint4*>(q + r * K_ROW + d) = make_uint4(0, 0, 0, 0);
                *reinterpret_cast<uint4*>(k + r * K_ROW + d) = make_uint4(0, 0, 0, 0);
            }
        }
        for (int i = threadIdx.x; i < C * v_pieces; i += 32 * W) {
            const int r = i / v_pieces, d = (i - r * v_pieces) * 8;
            if (r < count) ret_copy_async16(v + r * V_ROW + d, src + (size_t)r * p.proj_stride + p.v_off + h * vdim + v0 + d);
            else *reinterpret_cast<uint4*>(v + r * V_ROW + d) = make_uint4(0, 0, 0, 0);
        }
    };
    stage(0);

    // S[j]: value columns g and g + 8 of the warp's 16, keys 8 j + 2 t and the next
    float S[DIM / 8][4];
    const int va = v0 + 16 * warp + g, vb = va + 8;
#pragma unroll
    for (int j = 0; j < DIM / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int d = 8 * j + 2 * t + (e & 1), v = e < 2 ? va : vb;
            S[j][e] = (d < dim && v < vdim) ? s_in[(size_t)d * vdim + v] : 0.f;
        }

    for (int n = 0; n < chunks; ++n) {
        const int count = min(C, n_tok - n * C);
        const bf16* q = tiles + (n & 1) * STAGE;
        const bf16* k = q + C * K_ROW;
        const bf16* v = k + C * K_ROW;
        ret_copies_wait();
        __syncthreads();                               // the chunk is here for every thread; nobody reads the other stage or the scores
        if (n + 1 < chunks) stage(n + 1);
        for (int j = threadIdx.x; j < C; j += 32 * W) s_w[j] = j < count ? p.k_scale * s_pow[count - 1 - j] : 0.f;
        // -- decayed scores: a warp takes runs of 16 queries, up to the run's last key
        for (int rb = warp; rb < C / 16; rb += W) {
            float acc[C / 8][4];
#pragma unroll
            for (int j = 0; j < C / 8; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
#pragma unroll
            for (int ks = 0; ks < DIM / 16; ++ks) {
                uint32_t a[4];
                ret_matrices(a, q + (16 * rb + (m8 & 1) * 8 + r8) * K_ROW + 16 * ks + (m8 >> 1) * 8);
#pragma unroll
                for (int j = 0; j < C / 16; ++j) {
                    if (j <= rb) {
                        uint32_t bm[4];
                        ret_matrices(bm, k + (16 * j + (m8 >> 1) * 8 + r8) * K_ROW + 16 * ks + (m8 & 1) * 8);
                        ret_mma(acc[2 * j], a, bm[0], bm[1]);
                        ret_mma(acc[2 * j + 1], a, bm[2], bm[3]);
                    }
                }
            }
#pragma unroll
            for (int j = 0; j < C / 8; ++j) {
                if (j <= 2 * rb + 1) {
#pragma unroll
                    for (int half = 0; half < 2; ++half) {
                        const int i = 16 * rb + g + 8 * half, key = 8 * j + 2 * t;
                        const float x = key <= i ? acc[j][2 * half] * (p.k_scale * s_pow[i - key]) : 0.f;
                        const float y = key + 1 <= i ? acc[j][2 * half + 1] * (p.k_scale * s_pow[i - key - 1]) : 0.f;
                        uint32_t part[3];
                        ret_split(x, y, part);
#pragma unroll
                        for (int s = 0; s < 3; ++s) *reinterpret_cast<uint32_t*>(s_p + s * P_PART + i * P_ROW + key) = part[s];
                    }
                }
            }
        }
        __syncthreads();
        // -- o^T [16 value columns][C tokens]: what came before the chunk, then the chunk's own pairs
        float o[C / 8][4];
#pragma unroll
        for (int j = 0; j < C / 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) o[j][e] = 0.f;
#pragma unroll
        for (int ks = 0; ks < DIM / 16; ++ks) {
            uint32_t a[3][4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                uint32_t part[3];
                ret_split(S[2 * ks + (i >> 1)][2 * (i & 1)], S[2 * ks + (i >> 1)][2 * (i & 1) + 1], part);
#pragma unroll
                for (int s = 0; s < 3; ++s) a[s][i] = part[s];
            }
#pragma unroll
            for (int j = 0; j < C / 16; ++j) {
                uint32_t bm[4];
                ret_matrices(bm, q + (16 * j + (m8 >> 1) * 8 + r8) * K_ROW + 16 * ks + (m8 & 1) * 8);
#pragma unroll
                for (int s = 0; s < 3; ++s) {
                    ret_mma(o[2 * j], a[s], bm[0], bm[1]);
                    ret_mma(o[2 * j + 1], a[s], bm[2], bm[3]);
                }
            }
        }
#pragma unroll
        for (int j = 0; j < C / 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) o[j][e] *= s_pow[8 * j + 2 * t + (e & 1) + 1];
        uint32_t weighed[C / 16][3][4];                // the decayed values of 16 tokens each, split
#pragma unroll
        for (int ks = 0; ks < C / 16; ++ks) {
            uint32_t vt[4];                            // V^T: value columns of the warp, tokens 16 ks ..
            ret_matrices_turned(vt, v + (16 * ks + (m8 >> 1) * 8 + r8) * V_ROW + 16 * warp + (m8 & 1) * 8);
#pragma unroll
            for (int j = ks; j < C / 16; ++j)
#pragma unroll
                for (int s = 0; s < 3; ++s) {
                    uint32_t bm[4];
                    ret_matrices(bm, s_p + s * P_PART + (16 * j + (m8 >> 1) * 8 + r8) * P_ROW + 16 * ks + (m8 & 1) * 8);
                    ret_mma(o[2 * j], vt, bm[0], bm[1]);
                    ret_mma(o[2 * j + 1], vt, bm[2], bm[3]);
                }
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int key = 16 * ks + (i >> 1) * 8 + 2 * t;
                uint32_t part[3];
                ret_split(ret_low(vt[i]) * s_w[key], ret_high(vt[i]) * s_w[key + 1], part);
#pragma unroll
                for (int s = 0; s < 3; ++s) weighed[ks][s][i] = part[s];
            }
        }
#pragma unroll
        for (int j = 0; j < C / 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int token = 8 * j + 2 * t + (e & 1), col = e < 2 ? va : vb;
                if (token < count && col < vdim) p.raw[((size_t)(row0 + n * C + token) * p.heads + h) * vdim + col] = o[j][e];
            }
        // -- the state: its decay, less one, and the chunk's own sum.  The tensor cores cut off what does not fit when they add
        // into an accumulator; added into the state itself, chunk after chunk, that would pull it down (1e-5 of it after 3,000
        // tokens), so the chunk's sum starts from zero and is added here.
        const float less = p.decays[((size_t)h * 2 + 1) * (C + 1) + count];
#pragma unroll
        for (int j0 = 0; j0 < DIM / 16; j0 += 2) {
            float u[4][4];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) u[i][e] = 0.f;
#pragma unroll
            for (int ks = 0; ks < C / 16; ++ks) {
                uint32_t bm[2][4];
#pragma unroll
                for (int i = 0; i < 2; ++i)
                    ret_matrices_turned(bm[i], k + (16 * ks + (m8 & 1) * 8 + r8) * K_ROW + 16 * (j0 + i) + (m8 >> 1) * 8);
#pragma unroll
                for (int s = 2; s >= 0; --s)
#pragma unroll
                    for (int i = 0; i < 4; ++i) ret_mma(u[i], weighed[ks][s], bm[i >> 1][2 * (i & 1)], bm[i >> 1][2 * (i & 1) + 1]);
            }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) S[2 * j0 + i][e] = fmaf(less, S[2 * j0 + i][e], S[2 * j0 + i][e]) + u[i][e];
        }
    }
#pragma unroll
    for (int j = 0; j < DIM / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int d = 8 * j + 2 * t + (e & 1), col = e < 2 ? va : vb;
            if (d < dim && col < vdim) s_out[(size_t)d * vdim + col] = S[j][e];
        }
}

// Prompts with a bfloat16 projection: heads of up to 128 keys, sizes in steps of eight.
static int launch_retention_chunks(RetentionParams p, int num_rows, int num_seqs, cudaStream_t stream) {
    FRB_CHECK_ARG(p.dim % 8 == 0 && p.dim <= 128 && p.vdim % 8 == 0, "retention: heads of %d x %d are not the tensor-core kernel's", p.dim, p.vdim);
    FRB_CHECK_ARG(p.proj_stride % 8 == 0 && p.q_off % 8 == 0 && p.k_off % 8 == 0 && p.v_off % 8 == 0 && ((uintptr_t)p.proj & 15) == 0 && p.raw,
                  "retention: rows of %d entries do not lie on 16 bytes, or the outputs' buffer is missing", p.proj_stride);
    // four warps a block (64 value columns); two where that leaves SMs without a block
    const int slices = (p.vdim + 63) / 64;
    const bool narrow = p.vdim <= 32 || (long)num_seqs * p.heads * slices * 2 <= frb_dependent_launch_blocks();
    const int w = narrow ? 2 : 4, vs = 16 * w;
    const dim3 grid(num_seqs, p.heads, (p.vdim + vs - 1) / vs);
    FRB_CHECK_ARG(grid.z <= 65535, "retention: %d value columns exceed the grid", p.vdim);
#define FRB_RET_CHUNKS(DIM, W)                                                                                          \
    do {                                                                                                                \
        constexpr size_t smem = (2 * (size_t)RET_CHUNK * (2 * (DIM + RET_PAD) + 16 * W + RET_PAD) +                     \
                                 3 * (size_t)RET_CHUNK * (RET_CHUNK + RET_PAD)) * sizeof(bf16) + (2 * RET_CHUNK + 1) * sizeof(float); \
        auto kernel = retention_chunk_kernel<DIM, W>;                                                                   \
        cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                           \
        launch_dependent(kernel, grid, dim3(32 * W), smem, stream, p);                                                  \
    } while (0)
    if (p.dim <= 32) { if (w == 2) FRB_RET_CHUNKS(32, 2); else FRB_RET_CHUNKS(32, 4); }
    else if (p.dim <= 64) { if (w == 2) FRB_RET_CHUNKS(64, 2); else FRB_RET_CHUNKS(64, 4); }
    else { if (w == 2) FRB_RET_CHUNKS(128, 2); else FRB_RET_CHUNKS(128, 4); }
#undef FRB_RET_CHUNKS
    launch_dependent(retention_output_kernel<bf16, bf16>, dim3((num_rows * p.heads + 3) / 4), dim3(128), 0, stream, p, num_rows);
    FRB_RETURN_LAUNCH("retention");
}

// proj_dtype bfloat16: prompts, chunk by chunk on tensor cores (with out_dtype bfloat16); float32: token by token.
FRB_API int frb_retention(const void* proj, int proj_dtype, int proj_stride, int q_off, int k_off, int v_off, int g_off, const float* decays,
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
    if (proj_dtype == FRB_BF16) {
        FRB_CHECK_ARG(out_dtype == FRB_BF16, "retention: a bfloat16 projection with float32 outputs");
        p.raw = raw;
        return launch_retention_chunks(p, num_rows, num_seqs, stream);
    }
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
            launch_dependent(retention_output_kernel<OutT, float>, dim3((num_rows * heads + 3) / 4), dim3(128), 0, stream, p, num_rows);
    });
#undef FRB_RET
    FRB_RETURN_LAUNCH("retention");
}
