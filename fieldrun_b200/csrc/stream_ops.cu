// Operations on whole rows of the float32 residual stream that need no statistics, or only a row's mean square:
//
//   dyt_norm     the dynamic-tanh norm, y = tanh(alpha v) * w + b, of v = x + updates, for up to two norms of the same
//                v at once (a block whose two sublayers read the same x), with the sum stored back into x;
//                the updates are up to two float32 tensors and the weighted rows of routed experts, added in a
//                fixed order: x + ((d0 + d1) + sum over ranks of weight * row)
//   dyt_rows     the same norm for one norm without experts, several rows a thread, with a vector that every row gets and,
//                behind the norm, a token shift: out_t = h_t + (h_(t-1) - h_t) * share, the row before a step's first one
//                coming from the sequence's state; also the shift alone, of rows that another norm made
//   map_difference  two attention maps' outputs per head: a1 - lambda a2 over its root mean square, times a constant
//   rms_blend    out = share * (a / rms(a) * wa + b / rms(b) * wb), two mixers' outputs side by side
//   concat_rows  out = [a | b] row by row in the model dtype (a may get an update added first)
//   add_row_vector  out = y + vec, the same vector on every row
#include "common.cuh"

#define ROW_BLOCK 256
#define DYT_MAX_ROWS 64      // the most weighted rows that the norm sums for a token

struct DytParams {
    float* x;                 // [T, width]
    const float* delta0;      // [T, width] or null
    const float* delta1;      // [T, width] or null
    const float* y;           // [N, width] or null: expert outputs
    const float* ew;          // [T, top_k]
    const int* rowmap;        // [T * top_k]
    const int* rows;          // [R] or null: the rows to norm
    const float *w1, *b1, *alpha1;
    void* out1;
    const float *w2, *b2, *alpha2;   // null: one norm only
    void* out2;
    float* out2_32;           // null, or the second norm's result in float32 as well
    int top_k, width, write_back;
};

template <typename OutT>
__global__ void __launch_bounds__(ROW_BLOCK) dyt_norm_kernel(DytParams p) {
    __shared__ float s_weight[DYT_MAX_ROWS];
    __shared__ int s_row[DYT_MAX_ROWS];
    after_previous_kernel();
    const int r = blockIdx.x;
    const int src = p.rows ? p.rows[r] : r;
    const size_t base = (size_t)src * p.width, obase = (size_t)r * p.width;
    const float a1 = *p.alpha1, a2 = p.w2 ? *p.alpha2 : 0.f;
    if (p.y) {                                          // the row's experts: weights and rows once, not per element
        if (threadIdx.x < p.top_k) {
            s_weight[threadIdx.x] = p.ew[(size_t)src * p.top_k + threadIdx.x];
            s_row[threadIdx.x] = p.rowmap[(size_t)src * p.top_k + threadIdx.x];
        }
        __syncthreads();
    }
    for (int i = threadIdx.x; i < p.width; i += ROW_BLOCK) {
        float v = p.x[base + i];
        float d = 0.f;
        bool any = false;
        if (p.delta0) { d = p.delta0[base + i]; any = true; }
        if (p.delta1) { d += p.delta1[base + i]; any = true; }
        if (p.y) {
            float e = 0.f;
            for (int k = 0; k < p.top_k; ++k) e += s_weight[k] * p.y[(size_t)s_row[k] * p.width + i];
            d += e;
            any = true;
        }
        if (any) {
            v += d;
            if (p.write_back) p.x[base + i] = v;
        }
        ((OutT*)p.out1)[obase + i] = from_f32<OutT>(tanhf(a1 * v) * p.w1[i] + p.b1[i]);
        if (p.w2) {
            const float o2 = tanhf(a2 * v) * p.w2[i] + p.b2[i];
            ((OutT*)p.out2)[obase + i] = from_f32<OutT>(o2);
            if (p.out2_32) p.out2_32[obase + i] = o2;
        }
    }
}

FRB_API int frb_dyt_norm(float* x, const float* delta0, const float* delta1, const float* y, const float* ew,
                         const int* rowmap, int top_k, const int* rows, const float* w1, const float* b1,
                         const float* alpha1, void* out1, const float* w2, const float* b2, const float* alpha2, void* out2,
                         float* out2_32, int out_dtype, int num_rows, int width, int write_back, cudaStream_t stream) {
    if (num_rows == 0) return 0;
    FRB_CHECK_ARG(!(rows && write_back), "dyt_norm: chosen rows cannot be stored back");
    FRB_CHECK_ARG(!y || (top_k >= 1 && top_k <= DYT_MAX_ROWS), "dyt_norm: %d weighted rows a token are outside 1..%d", top_k, DYT_MAX_ROWS);
    DytParams p;
    p.x = x; p.delta0 = delta0; p.delta1 = delta1; p.y = y; p.ew = ew; p.rowmap = rowmap; p.rows = rows;
    p.w1 = w1; p.b1 = b1; p.alpha1 = alpha1; p.out1 = out1; p.w2 = w2; p.b2 = b2; p.alpha2 = alpha2; p.out2 = out2;
    p.out2_32 = out2_32; p.top_k = top_k; p.width = width; p.write_back = write_back;
    FRB_DISPATCH_DTYPE(out_dtype, OutT, {
        launch_dependent(dyt_norm_kernel<OutT>, dim3(num_rows), dim3(ROW_BLOCK), 0, stream, p);
    });
    FRB_RETURN_LAUNCH("dyt_norm");
}

// ---------------------------------------------------------------------------------------------------- dyt_rows

struct DytRowsParams {
    const float* x;           // [T, width]
    const float* delta0;      // [T, width] or null
    const float* delta1;      // [T, width] or null
    const float* vec;         // [width] or null: added to every row
    const int* rows;          // [R] or null: the rows to norm (without shift)
    const float *w, *b, *alpha;
    float* stream;            // [T, width] or null: gets x + updates; with a shift never x itself (a row is read again by the next one)
    void* out;                // [R, width]
    int width, num_rows, rows_per_thread;
    // the shift
    const float* share;       // [width]
    const int *tok_seq, *seq_slot, *seq_start, *cu_q_len;
    float* state;             // [slots][2][copy_floats], this part's at state_offset
    long long copy_floats, state_offset;
};

template <int V> struct Floats { float v[V]; };
template <int V> __device__ __forceinline__ Floats<V> load_floats(const float* p);
template <> __device__ __forceinline__ Floats<1> load_floats<1>(const float* p) { return {{*p}}; }
template <> __device__ __forceinline__ Floats<4> load_floats<4>(const float* p) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    return {{f.x, f.y, f.z, f.w}};
}
template <int V> __device__ __forceinline__ void store_floats(float* p, const Floats<V>& f);
template <> __device__ __forceinline__ void store_floats<1>(float* p, const Floats<1>& f) { *p = f.v[0]; }
template <> __device__ __forceinline__ void store_floats<4>(float* p, const Floats<4>& f) {
    *reinterpret_cast<float4*>(p) = make_float4(f.v[0], f.v[1], f.v[2], f.v[3]);
}
template <typename T, int V> __device__ __forceinline__ void store_typed(T* p, const Floats<V>& f) {
    if constexpr (sizeof(T) == 4) {
        store_floats<V>((float*)p, f);
    } else if constexpr (V == 1) {
        *p = from_f32<T>(f.v[0]);
    } else {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(f.v[0], f.v[1]), hi = __floats2bfloat162_rn(f.v[2], f.v[3]);
        uint2 raw;
        raw.x = *reinterpret_cast<const unsigned int*>(&lo);
        raw.y = *reinterpret_cast<const unsigned int*>(&hi);
        *reinterpret_cast<uint2*>(p) = raw;
    }
}

#define DYT_ROWS_AT_ONCE 4   // rows whose inputs a thread asks for before it uses the first

// A thread takes V columns of rows_per_thread neighbouring rows.  NORM: dynamic tanh of x + updates (else x holds normed rows
// already).  SHIFT: the previous row's h stays in registers; before the thread's first row it is made again from that row's
// inputs, or comes from the state if the row opens its sequence's new tokens.  The thread of a sequence's first new row also
// writes the new state, from the last new row's inputs, after it has read the old one: a step of several tokens may read and
// write the same copy.
template <typename OutT, int V, bool NORM, bool SHIFT>
__global__ void __launch_bounds__(128) dyt_rows_kernel(DytRowsParams p) {
    after_previous_kernel();
    const int c = (blockIdx.y * 128 + threadIdx.x) * V;
    if (c >= p.width) return;
    const int r_begin = blockIdx.x * p.rows_per_thread, r_end = min(p.num_rows, r_begin + p.rows_per_thread);
    Floats<V> w, bias, vec, share;
    float alpha = 0.f;
    if (NORM) { w = load_floats<V>(p.w + c); bias = load_floats<V>(p.b + c); alpha = *p.alpha; }
    if (SHIFT) share = load_floats<V>(p.share + c);
#pragma unroll
    for (int e = 0; e < V; ++e) vec.v[e] = 0.f;
    if (p.vec) vec = load_floats<V>(p.vec + c);
    const bool updates = p.delta0 || p.delta1 || p.vec;
    const bool two = p.delta1 != nullptr;

    auto sum_of = [&](const Floats<V>& x, const Floats<V>& d0, const Floats<V>& d1) {
        Floats<V> v = x;
        if (updates) {
#pragma unroll
            for (int e = 0; e < V; ++e) v.v[e] = x.v[e] + ((d0.v[e] + d1.v[e]) + vec.v[e]);
        }
        return v;
    };
    auto normed = [&](const Floats<V>& v) {
        if (!NORM) return v;
        Floats<V> h;
#pragma unroll
        for (int e = 0; e < V; ++e) h.v[e] = fmaf(tanhf(alpha * v.v[e]), w.v[e], bias.v[e]);
        return h;
    };
    Floats<V> zero;
#pragma unroll
    for (int e = 0; e < V; ++e) zero.v[e] = 0.f;
    auto h_of_row = [&](int r) {
        const size_t at = (size_t)r * p.width + c;
        const Floats<V> x = load_floats<V>(p.x + at);
        const Floats<V> d0 = p.delta0 ? load_floats<V>(p.delta0 + at) : zero, d1 = two ? load_floats<V>(p.delta1 + at) : zero;
        return normed(sum_of(x, d0, d1));
    };

    Floats<V> before = zero;
    int next_start = -1;                                  // the row that opens the next sequence of the step
    int seq = 0;
    if (SHIFT) {
        seq = p.tok_seq[r_begin];
        next_start = p.cu_q_len[seq];
        if (r_begin > next_start) {
            before = h_of_row(r_begin - 1);
            next_start = p.cu_q_len[++seq];
        }
    }
    for (int r0 = r_begin; r0 < r_end; r0 += DYT_ROWS_AT_ONCE) {
        Floats<V> x[DYT_ROWS_AT_ONCE], d0[DYT_ROWS_AT_ONCE], d1[DYT_ROWS_AT_ONCE];
#pragma unroll
        for (int q = 0; q < DYT_ROWS_AT_ONCE; ++q) {
            x[q] = d0[q] = d1[q] = zero;
            if (r0 + q < r_end) {
                const size_t at = (size_t)((!SHIFT && p.rows) ? p.rows[r0 + q] : r0 + q) * p.width + c;
                x[q] = load_floats<V>(p.x + at);
                if (p.delta0) d0[q] = load_floats<V>(p.delta0 + at);
                if (two) d1[q] = load_floats<V>(p.delta1 + at);
            }
        }
#pragma unroll
        for (int q = 0; q < DYT_ROWS_AT_ONCE; ++q) {
            const int r = r0 + q;
            if (r >= r_end) break;
            const Floats<V> v = sum_of(x[q], d0[q], d1[q]);
            const Floats<V> h = normed(v);
            if (p.stream) store_floats<V>(p.stream + (size_t)r * p.width + c, v);
            Floats<V> y = h;
            if (SHIFT) {
                if (r == next_start) {                    // this row opens sequence `seq`
                    const int n = p.cu_q_len[seq + 1] - r, start = p.seq_start[seq];
                    float* state = p.state + (size_t)p.seq_slot[seq] * 2 * p.copy_floats + p.state_offset + c;
                    before = load_floats<V>(state + (start & 1) * p.copy_floats);
                    const Floats<V> last = n == 1 ? h : h_of_row(r + n - 1);
                    store_floats<V>(state + ((start + n) & 1) * p.copy_floats, last);
                    next_start = r + n;
                    ++seq;
                }
#pragma unroll
                for (int e = 0; e < V; ++e) y.v[e] = fmaf(before.v[e] - h.v[e], share.v[e], h.v[e]);
                before = h;
            }
            store_typed<OutT, V>((OutT*)p.out + (size_t)r * p.width + c, y);
        }
    }
}

FRB_API int frb_dyt_rows(const float* x, const float* delta0, const float* delta1, const float* vec, const int* rows,
                         const float* w, const float* b, const float* alpha, float* stream_out, void* out, int out_dtype,
                         int num_rows, int width, const float* share, const int* tok_seq, const int* seq_slot,
                         const int* seq_start, const int* cu_q_len, float* state, long long copy_floats, long long state_offset,
                         cudaStream_t stream) {
    if (num_rows == 0) return 0;
    const bool norm = w != nullptr, shift = share != nullptr;
    FRB_CHECK_ARG(!(rows && (stream_out || shift)), "dyt_rows: chosen rows are neither stored back nor shifted");
    FRB_CHECK_ARG(!shift || (tok_seq && seq_slot && seq_start && cu_q_len && state && stream_out != x), "dyt_rows: a shift needs the step's tables, "
                  "a state and a buffer of its own for the stream");
    FRB_CHECK_ARG(norm || shift, "dyt_rows: neither a norm nor a shift");
    DytRowsParams p;
    p.x = x; p.delta0 = delta0; p.delta1 = delta1; p.vec = vec; p.rows = rows; p.w = w; p.b = b; p.alpha = alpha;
    p.stream = stream_out; p.out = out; p.width = width; p.num_rows = num_rows;
    p.share = share; p.tok_seq = tok_seq; p.seq_slot = seq_slot; p.seq_start = seq_start; p.cu_q_len = cu_q_len;
    p.state = state; p.copy_floats = copy_floats; p.state_offset = state_offset;
    const auto on16 = [](const void* ptr) { return ((uintptr_t)ptr & 15) == 0; };
    const bool by_four = width % 4 == 0 && copy_floats % 4 == 0 && state_offset % 4 == 0 && on16(x) && on16(delta0) && on16(delta1) &&
                         on16(vec) && on16(w) && on16(b) && on16(stream_out) && on16(out) && on16(share) && on16(state);
    // many rows: a thread takes eight (the row before is normed once more per run); few: one, for more threads
    p.rows_per_thread = num_rows >= 1024 ? 8 : num_rows >= 512 ? 4 : 1;
    const int columns = 128 * (by_four ? 4 : 1);
    dim3 grid((num_rows + p.rows_per_thread - 1) / p.rows_per_thread, (width + columns - 1) / columns);
    FRB_CHECK_ARG(grid.y <= 65535, "dyt_rows: rows of %d exceed the grid", width);
#define FRB_DYT_ROWS(V)                                                                                              \
    do {                                                                                                             \
        auto kernel = !norm ? dyt_rows_kernel<OutT, V, false, true>                                                  \
                            : shift ? dyt_rows_kernel<OutT, V, true, true> : dyt_rows_kernel<OutT, V, true, false>;  \
        launch_dependent(kernel, grid, dim3(128), 0, stream, p);                                                     \
    } while (0)
    FRB_DISPATCH_DTYPE(out_dtype, OutT, {
        if (by_four) FRB_DYT_ROWS(4); else FRB_DYT_ROWS(1);
    });
#undef FRB_DYT_ROWS
    FRB_RETURN_LAUNCH("dyt_rows");
}

// ---------------------------------------------------------------------------------------------------- map_difference

// maps [T, kv_heads, 2, group, vd] float32: o = map 1 - lam * map 2 of a head, out [T, heads, vd] = o / sqrt(mean(o^2) + eps) *
// factor.  A warp per (token, head).
template <typename OutT>
__global__ void __launch_bounds__(ROW_BLOCK) map_difference_kernel(const float* __restrict__ maps, const float* __restrict__ lam,
                                                                   OutT* __restrict__ out, long long items, int heads, int group,
                                                                   int vd, float eps, float factor) {
    after_previous_kernel();
    const int lane = threadIdx.x & 31;
    const long long item = (long long)blockIdx.x * (ROW_BLOCK / 32) + (threadIdx.x >> 5);
    if (item >= items) return;
    const long long t = item / heads;
    const int head = (int)(item - t * heads), g = head / group, r = head - g * group;
    const float* a1 = maps + ((t * heads + (long long)g * group) * 2 + r) * vd;
    const float* a2 = a1 + (long long)group * vd;
    const float l = *lam;
    float ss = 0.f;
    for (int d = lane; d < vd; d += 32) {
        const float o = a1[d] - l * a2[d];
        ss += o * o;
    }
    const float scale = factor / sqrtf(warp_sum(ss) / (float)vd + eps);
    for (int d = lane; d < vd; d += 32) out[item * vd + d] = from_f32<OutT>((a1[d] - l * a2[d]) * scale);
}

FRB_API int frb_map_difference(const float* maps, const float* lam, void* out, int out_dtype, int num_rows, int heads, int kv_heads,
                               int vd, float eps, float factor, cudaStream_t stream) {
    if (num_rows == 0) return 0;
    FRB_CHECK_ARG(kv_heads >= 1 && heads % kv_heads == 0, "map_difference: %d heads over %d value heads", heads, kv_heads);
    const long long items = (long long)num_rows * heads;
    FRB_DISPATCH_DTYPE(out_dtype, OutT, {
        launch_dependent(map_difference_kernel<OutT>, dim3((unsigned)((items + ROW_BLOCK / 32 - 1) / (ROW_BLOCK / 32))), dim3(ROW_BLOCK), 0,
                         stream, maps, lam, (OutT*)out, items, heads, heads / kv_heads, vd, eps, factor);
    });
    FRB_RETURN_LAUNCH("map_difference");
}

// ---------------------------------------------------------------------------------------------------- rms_blend

__global__ void __launch_bounds__(ROW_BLOCK) rms_blend_kernel(const float* __restrict__ a, const float* __restrict__ b,
                                                              const float* __restrict__ wa, const float* __restrict__ wb,
                                                              float* __restrict__ out, int width, float eps, float share) {
    __shared__ float scratch[64];
    after_previous_kernel();
    const size_t base = (size_t)blockIdx.x * width;
    float sa = 0.f, sb = 0.f;
    for (int i = threadIdx.x; i < width; i += ROW_BLOCK) {
        const float va = a[base + i], vb = b[base + i];
        sa += va * va;
        sb += vb * vb;
    }
    block_sum_pair<ROW_BLOCK>(sa, sb, scratch);
    const float ra = 1.0f / sqrtf(sa / (float)width + eps), rb = 1.0f / sqrtf(sb / (float)width + eps);
    for (int i = threadIdx.x; i < width; i += ROW_BLOCK)
        out[base + i] = share * (a[base + i] * ra * wa[i] + b[base + i] * rb * wb[i]);
}

FRB_API int frb_rms_blend(const float* a, const float* b, const float* wa, const float* wb, float* out, int num_rows,
                          int width, float eps, float share, cudaStream_t stream) {
    if (num_rows == 0) return 0;
    launch_dependent(rms_blend_kernel, dim3(num_rows), dim3(ROW_BLOCK), 0, stream, a, b, wa, wb, out, width, eps, share);
    FRB_RETURN_LAUNCH("rms_blend");
}

// ---------------------------------------------------------------------------------------------------- concat, add

template <typename OutT>
__global__ void __launch_bounds__(ROW_BLOCK) concat_rows_kernel(float* a, const float* __restrict__ delta,
                                                                const float* __restrict__ b, OutT* __restrict__ out, int wa,
                                                                int wb) {
    after_previous_kernel();
    const size_t r = blockIdx.x;
    for (int i = threadIdx.x; i < wa + wb; i += ROW_BLOCK) {
        float v;
        if (i < wa) {
            v = a[r * wa + i];
            if (delta) v += delta[r * wa + i];
        } else {
            v = b[r * wb + i - wa];
        }
        out[r * (wa + wb) + i] = from_f32<OutT>(v);
    }
}

FRB_API int frb_concat_rows(float* a, const float* delta, const float* b, void* out, int out_dtype, int num_rows, int wa,
                            int wb, cudaStream_t stream) {
    if (num_rows == 0) return 0;
    FRB_DISPATCH_DTYPE(out_dtype, OutT, {
        launch_dependent(concat_rows_kernel<OutT>, dim3(num_rows), dim3(ROW_BLOCK), 0, stream, a, delta, b, (OutT*)out, wa, wb);
    });
    FRB_RETURN_LAUNCH("concat_rows");
}

__global__ void __launch_bounds__(ROW_BLOCK) add_row_vector_kernel(const float* __restrict__ y, const float* __restrict__ vec,
                                                                   float* __restrict__ out, int width) {
    after_previous_kernel();
    const size_t base = (size_t)blockIdx.x * width;
    for (int i = threadIdx.x; i < width; i += ROW_BLOCK) out[base + i] = y[base + i] + vec[i];
}

FRB_API int frb_add_row_vector(const float* y, const float* vec, float* out, int num_rows, int width, cudaStream_t stream) {
    if (num_rows == 0) return 0;
    launch_dependent(add_row_vector_kernel, dim3(num_rows), dim3(ROW_BLOCK), 0, stream, y, vec, out, width);
    FRB_RETURN_LAUNCH("add_row_vector");
}

// out[t, h * vd + d] *= sigmoid(gate[t * stride + h]): a gate per token and head on an attention's output
template <typename T>
__global__ void __launch_bounds__(ROW_BLOCK) head_gate_kernel(T* __restrict__ out, const float* __restrict__ gate, int stride,
                                                              int heads, int vd) {
    after_previous_kernel();
    const size_t t = blockIdx.x;
    for (int i = threadIdx.x; i < heads * vd; i += ROW_BLOCK) {
        const float g = 1.0f / (1.0f + expf(-gate[t * stride + i / vd]));
        out[t * heads * vd + i] = from_f32<T>(to_f32<T>(out[t * heads * vd + i]) * g);
    }
}

FRB_API int frb_head_gate(void* out, int dtype, const float* gate, int stride, int num_rows, int heads, int vd,
                          cudaStream_t stream) {
    if (num_rows == 0) return 0;
    FRB_DISPATCH_DTYPE(dtype, T, {
        launch_dependent(head_gate_kernel<T>, dim3(num_rows), dim3(ROW_BLOCK), 0, stream, (T*)out, gate, stride, heads, vd);
    });
    FRB_RETURN_LAUNCH("head_gate");
}

// ---------------------------------------------------------------------------------------------------- weighted_pair

// out = ca * a + cb * b: two mixers' outputs side by side, each with a constant weight.
__global__ void __launch_bounds__(ROW_BLOCK) weighted_pair_kernel(const float* __restrict__ a, const float* __restrict__ b,
                                                                  float* __restrict__ out, size_t total, float ca, float cb) {
    after_previous_kernel();
    const size_t i = (size_t)blockIdx.x * ROW_BLOCK + threadIdx.x;
    if (i < total) out[i] = ca * a[i] + cb * b[i];
}

FRB_API int frb_weighted_pair(const float* a, const float* b, float* out, long long total, float ca, float cb, cudaStream_t stream) {
    if (total == 0) return 0;
    launch_dependent(weighted_pair_kernel, dim3((unsigned)((total + ROW_BLOCK - 1) / ROW_BLOCK)), dim3(ROW_BLOCK), 0, stream, a, b, out,
                     (size_t)total, ca, cb);
    FRB_RETURN_LAUNCH("weighted_pair");
}
