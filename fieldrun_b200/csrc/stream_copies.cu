// Hyper-connections: a residual stream kept as S copies of a row (x_1 .. x_S, float32).  A sublayer f reads a weighted sum
// of the copies and its output is spread over all of them:
//
//   u = sum_s in[s] x_s;   y = f(norm(u));   x_t <- sum_s mix[s, t] x_s + out[t] y            (all copies at once)
//
// One kernel does what lies between two sublayers in one pass over the rows: the update of the copies by up to two outputs
//
//   v_t = sum_s mix[s, t] x_s + oa[t] ya + ob[t] yb,     yb = (d0 + d1) + sum over ranks r of weight[r] * row[r]
//
// (routed experts' rows in rank order), stored when `x_out` is given, then u = sum_t in[t] v_t and its dynamic-tanh norm
// tanh(alpha u) * w + b.  Both steps are linear in x, ya and yb, so a pass that does not store the copies never makes them: it
// takes u = sum_s c_s x_s + ca ya + cb yb with c = mix in, ca = oa . in, cb = ob . in.  That is how the copies are left as
// they are between a layer's two sublayers, and stored once a layer with the product of the two mixes: at S = 4 a layer
// moves 15 rows of float32 per token instead of 18.
//
// Nothing crosses columns: a thread owns V neighbouring columns of all copies of a row, and storing over x itself is safe.
// All sums are float32, in an order that depends on S alone.
#include "common.cuh"

#define COPIES_BLOCK 128
#define COPIES_MAX_STREAMS 64
#define COPIES_MAX_TOP_K 64
#define COPIES_MAX_ROWS 8          // most rows a block takes

struct CopiesParams {
    const float* x;           // [T, S, width], or [T, width] standing for S equal copies
    long long x_row, x_copy;  // floats from row to row and from copy to copy (0: equal copies)
    float* x_out;             // [T, S, width] or null
    const float *ya, *oa;     // [T, width], [S] or null
    const float *d0, *d1;     // [T, width] or null: parts of yb
    const float* y;           // [N, width] or null: expert outputs
    const float* ew;          // [T, top_k]
    const int* rowmap;        // [T * top_k]
    const float* ob;          // [S]
    const float* mix;         // [S, S] or null: the copies as they are
    const float* in;          // [S] or null: ones
    const int* rows;          // [R] or null: the rows to take
    const float *w, *b, *alpha;   // null: u itself is the result
    void* out;                // [R, width] or null
    float* out32;             // [R, width] or null
    int streams, top_k, width, num_rows, rows_per_block;
};

template <int V> struct Columns { float v[V]; };
template <int V> __device__ __forceinline__ Columns<V> load_columns(const float* p) {
    Columns<V> c;
    if constexpr (V == 4) {
        const float4 f = *reinterpret_cast<const float4*>(p);
        c.v[0] = f.x; c.v[1] = f.y; c.v[2] = f.z; c.v[3] = f.w;
    } else {
        c.v[0] = *p;
    }
    return c;
}
template <int V, typename T> __device__ __forceinline__ void store_columns(T* p, const Columns<V>& c) {
    if constexpr (V == 1) {
        *p = from_f32<T>(c.v[0]);
    } else if constexpr (sizeof(T) == 4) {
        *reinterpret_cast<float4*>(p) = make_float4(c.v[0], c.v[1], c.v[2], c.v[3]);
    } else {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(c.v[0], c.v[1]), hi = __floats2bfloat162_rn(c.v[2], c.v[3]);
        uint2 raw;
        raw.x = *reinterpret_cast<const unsigned int*>(&lo);
        raw.y = *reinterpret_cast<const unsigned int*>(&hi);
        *reinterpret_cast<uint2*>(p) = raw;
    }
}

// A row's experts, fetched once per block.
struct RowExperts {
    float weight[COPIES_MAX_ROWS * COPIES_MAX_TOP_K];
    int row[COPIES_MAX_ROWS * COPIES_MAX_TOP_K];
};

__device__ __forceinline__ void fetch_experts(const CopiesParams& p, RowExperts& s, int r_begin, int count) {
    if (!p.y) return;
    for (int i = threadIdx.x; i < count * p.top_k; i += COPIES_BLOCK) {
        const int r = r_begin + i / p.top_k;
        const size_t at = (size_t)(p.rows ? p.rows[r] : r) * p.top_k + i % p.top_k;
        s.weight[i] = p.ew[at];
        s.row[i] = p.rowmap[at];
    }
    __syncthreads();
}

// The columns of yb of row src (row n of the block).
template <int V> __device__ __forceinline__ Columns<V> second_update(const CopiesParams& p, const RowExperts& s, int n, size_t at, int c) {
    Columns<V> sum;
#pragma unroll
    for (int e = 0; e < V; ++e) sum.v[e] = 0.f;
    if (p.d0) sum = load_columns<V>(p.d0 + at);
    if (p.d1) {
        const Columns<V> d = load_columns<V>(p.d1 + at);
#pragma unroll
        for (int e = 0; e < V; ++e) sum.v[e] += d.v[e];
    }
    if (p.y) {
        Columns<V> total;
#pragma unroll
        for (int e = 0; e < V; ++e) total.v[e] = 0.f;
        for (int k0 = 0; k0 < p.top_k; k0 += 4) {                    // four experts' rows on their way at a time
            Columns<V> part[4];
#pragma unroll
            for (int k = 0; k < 4; ++k)
                if (k0 + k < p.top_k) part[k] = load_columns<V>(p.y + (size_t)s.row[n * p.top_k + k0 + k] * p.width + c);
#pragma unroll
            for (int k = 0; k < 4; ++k)
                if (k0 + k < p.top_k) {
                    const float weight = s.weight[n * p.top_k + k0 + k];
#pragma unroll
                    for (int e = 0; e < V; ++e) total.v[e] = fmaf(weight, part[k].v[e], total.v[e]);
                }
        }
#pragma unroll
        for (int e = 0; e < V; ++e) sum.v[e] += total.v[e];
    }
    return sum;
}

template <typename OutT, int V>
__device__ __forceinline__ void finish(const CopiesParams& p, const Columns<V>& u, const Columns<V>& w, const Columns<V>& b, float alpha,
                                       size_t at) {
    Columns<V> h = u;
    if (p.w) {
#pragma unroll
        for (int e = 0; e < V; ++e) h.v[e] = fmaf(tanhf(alpha * u.v[e]), w.v[e], b.v[e]);
    }
    if (p.out) store_columns<V, OutT>((OutT*)p.out + at, h);
    if (p.out32) store_columns<V, float>(p.out32 + at, h);
}

// Up to MOST copies, held in registers.  STORE: the new copies are made and stored; else only their weighted sum.
template <typename OutT, int MOST, bool STORE>
__global__ void __launch_bounds__(COPIES_BLOCK) copies_kernel(CopiesParams p) {
    constexpr int V = 4;
    __shared__ float s_mix[MOST * MOST], s_a[MOST], s_b[MOST], s_in[MOST];
    __shared__ RowExperts experts;
    let_next_kernel_start();
    const int S = p.streams;
    // the constants are nobody's output: they are read while the kernel before this one still runs
    for (int i = threadIdx.x; i < S * S; i += COPIES_BLOCK) s_mix[i / S * MOST + i % S] = p.mix ? p.mix[i] : i / S == i % S ? 1.f : 0.f;
    if (threadIdx.x < S) {
        s_a[threadIdx.x] = p.oa ? p.oa[threadIdx.x] : 0.f;
        s_b[threadIdx.x] = p.ob ? p.ob[threadIdx.x] : 0.f;
        s_in[threadIdx.x] = p.in ? p.in[threadIdx.x] : 1.f;
    }
    const int c = (blockIdx.y * COPIES_BLOCK + threadIdx.x) * V;
    const bool mine = c < p.width;
    Columns<V> w, b;
    float alpha = 0.f;
    if (p.w && mine) { w = load_columns<V>(p.w + c); b = load_columns<V>(p.b + c); alpha = *p.alpha; }
    __syncthreads();
    float c_x[MOST], c_a = 0.f, c_b = 0.f;
    if (!STORE) {
#pragma unroll
        for (int s = 0; s < MOST; ++s) {
            c_x[s] = 0.f;
            if (s < S) {
                for (int t = 0; t < S; ++t) c_x[s] = fmaf(s_mix[s * MOST + t], s_in[t], c_x[s]);
                c_a = fmaf(s_a[s], s_in[s], c_a);
                c_b = fmaf(s_b[s], s_in[s], c_b);
            }
        }
    }
    wait_for_previous_kernel();
    const int r_begin = blockIdx.x * p.rows_per_block, count = min(p.rows_per_block, p.num_rows - r_begin);
    fetch_experts(p, experts, r_begin, count);
    if (!mine) return;
    const bool has_b = p.d0 || p.d1 || p.y;
    for (int n = 0; n < count; ++n) {
        const int r = r_begin + n;
        const int src = p.rows ? p.rows[r] : r;
        const size_t at = (size_t)src * p.width + c;
        const float* xs = p.x + (size_t)src * p.x_row + c;
        Columns<V> x[MOST], ya, yb;
#pragma unroll
        for (int s = 0; s < MOST; ++s)
            if (s < S) x[s] = load_columns<V>(xs + s * p.x_copy);
        if (p.ya) ya = load_columns<V>(p.ya + at);
        if (has_b) yb = second_update<V>(p, experts, n, at, c);
        Columns<V> u;
#pragma unroll
        for (int e = 0; e < V; ++e) u.v[e] = 0.f;
        if (STORE) {
            float* dst = p.x_out + (size_t)src * S * p.width + c;
#pragma unroll
            for (int t = 0; t < MOST; ++t)
                if (t < S) {
                    Columns<V> v;
#pragma unroll
                    for (int e = 0; e < V; ++e) v.v[e] = 0.f;
#pragma unroll
                    for (int s = 0; s < MOST; ++s)
                        if (s < S) {
                            const float m = s_mix[s * MOST + t];
#pragma unroll
                            for (int e = 0; e < V; ++e) v.v[e] = fmaf(m, x[s].v[e], v.v[e]);
                        }
                    if (p.ya) {
#pragma unroll
                        for (int e = 0; e < V; ++e) v.v[e] = fmaf(s_a[t], ya.v[e], v.v[e]);
                    }
                    if (has_b) {
#pragma unroll
                        for (int e = 0; e < V; ++e) v.v[e] = fmaf(s_b[t], yb.v[e], v.v[e]);
                    }
                    store_columns<V, float>(dst + (size_t)t * p.width, v);
#pragma unroll
                    for (int e = 0; e < V; ++e) u.v[e] = fmaf(s_in[t], v.v[e], u.v[e]);
                }
        } else {
#pragma unroll
            for (int s = 0; s < MOST; ++s)
                if (s < S) {
#pragma unroll
                    for (int e = 0; e < V; ++e) u.v[e] = fmaf(c_x[s], x[s].v[e], u.v[e]);
                }
            if (p.ya) {
#pragma unroll
                for (int e = 0; e < V; ++e) u.v[e] = fmaf(c_a, ya.v[e], u.v[e]);
            }
            if (has_b) {
#pragma unroll
                for (int e = 0; e < V; ++e) u.v[e] = fmaf(c_b, yb.v[e], u.v[e]);
            }
        }
        finish<OutT, V>(p, u, w, b, alpha, (size_t)r * p.width + c);
    }
}

// Any width and any number of copies up to COPIES_MAX_STREAMS: a column a thread, its copies in shared memory.
template <typename OutT>
__global__ void __launch_bounds__(COPIES_BLOCK) copies_any_kernel(CopiesParams p) {
    extern __shared__ float dynamic[];                   // mix [S, S], a [S], b [S], in [S], the columns [S][block]
    __shared__ RowExperts experts;
    let_next_kernel_start();
    const int S = p.streams;
    float *s_mix = dynamic, *s_a = s_mix + S * S, *s_b = s_a + S, *s_in = s_b + S, *columns = s_in + S + threadIdx.x;
    for (int i = threadIdx.x; i < S * S; i += COPIES_BLOCK) s_mix[i] = p.mix ? p.mix[i] : i / S == i % S ? 1.f : 0.f;
    for (int i = threadIdx.x; i < S; i += COPIES_BLOCK) {
        s_a[i] = p.oa ? p.oa[i] : 0.f;
        s_b[i] = p.ob ? p.ob[i] : 0.f;
        s_in[i] = p.in ? p.in[i] : 1.f;
    }
    const int c = blockIdx.y * COPIES_BLOCK + threadIdx.x;
    const bool mine = c < p.width;
    Columns<1> w, b;
    float alpha = 0.f;
    if (p.w && mine) { w = load_columns<1>(p.w + c); b = load_columns<1>(p.b + c); alpha = *p.alpha; }
    __syncthreads();
    wait_for_previous_kernel();
    const int r_begin = blockIdx.x * p.rows_per_block, count = min(p.rows_per_block, p.num_rows - r_begin);
    fetch_experts(p, experts, r_begin, count);
    if (!mine) return;
    for (int n = 0; n < count; ++n) {
        const int r = r_begin + n;
        const int src = p.rows ? p.rows[r] : r;
        const size_t at = (size_t)src * p.width + c;
        for (int s = 0; s < S; ++s) columns[s * COPIES_BLOCK] = p.x[(size_t)src * p.x_row + s * p.x_copy + c];
        const float ya = p.ya ? p.ya[at] : 0.f, yb = second_update<1>(p, experts, n, at, c).v[0];
        Columns<1> u = {{0.f}};
        for (int t = 0; t < S; ++t) {
            float v = 0.f;
            for (int s = 0; s < S; ++s) v = fmaf(s_mix[s * S + t], columns[s * COPIES_BLOCK], v);
            v = fmaf(s_a[t], ya, v);
            v = fmaf(s_b[t], yb, v);
            if (p.x_out) p.x_out[((size_t)src * S + t) * p.width + c] = v;
            u.v[0] = fmaf(s_in[t], v, u.v[0]);
        }
        finish<OutT, 1>(p, u, w, b, alpha, (size_t)r * p.width + c);
    }
}

FRB_API int frb_stream_copies(const float* x, int equal_copies, float* x_out, const float* ya, const float* oa, const float* d0,
                              const float* d1, const float* y, const float* ew, const int* rowmap, int top_k, const float* ob,
                              const float* mix, const float* in, const int* rows, const float* w, const float* b, const float* alpha,
                              void* out, int out_dtype, float* out32, int num_rows, int width, int streams, cudaStream_t stream) {
    if (num_rows == 0) return 0;
    FRB_CHECK_ARG(streams >= 1 && streams <= COPIES_MAX_STREAMS, "stream_copies: %d copies are outside 1..%d", streams, COPIES_MAX_STREAMS);
    FRB_CHECK_ARG(!y || (ew && rowmap && top_k >= 1 && top_k <= COPIES_MAX_TOP_K), "stream_copies: %d weighted rows a token are outside 1..%d",
                  top_k, COPIES_MAX_TOP_K);
    FRB_CHECK_ARG(!(rows && x_out), "stream_copies: chosen rows are not stored back");
    FRB_CHECK_ARG((!ya || oa) && (!(d0 || d1 || y) || ob), "stream_copies: an update without its weights on the copies");
    FRB_CHECK_ARG(!(x_out == x && equal_copies), "stream_copies: copies stored over the one row that stands for them");
    FRB_CHECK_ARG(out || out32, "stream_copies: nowhere to put the result");
    FRB_CHECK_ARG(!w || (b && alpha), "stream_copies: a norm without its bias or alpha");
    CopiesParams p;
    p.x = x; p.x_row = equal_copies ? width : (long long)streams * width; p.x_copy = equal_copies ? 0 : width; p.x_out = x_out;
    p.ya = ya; p.oa = oa; p.d0 = d0; p.d1 = d1; p.y = y; p.ew = ew; p.rowmap = rowmap; p.ob = ob; p.mix = mix; p.in = in; p.rows = rows;
    p.w = w; p.b = b; p.alpha = alpha; p.out = out; p.out32 = out32;
    p.streams = streams; p.top_k = y ? top_k : 0; p.width = width; p.num_rows = num_rows;
    const auto on16 = [](const void* ptr) { return ((uintptr_t)ptr & 15) == 0; };
    const bool by_four = streams <= 8 && width % 4 == 0 && on16(x) && on16(x_out) && on16(ya) && on16(d0) && on16(d1) && on16(y) && on16(w) &&
                         on16(b) && on16(out) && on16(out32);
    p.rows_per_block = num_rows >= 2048 ? 4 : num_rows >= 512 ? 2 : 1;
    const int columns = COPIES_BLOCK * (by_four ? 4 : 1);
    dim3 grid((num_rows + p.rows_per_block - 1) / p.rows_per_block, (width + columns - 1) / columns);
    FRB_CHECK_ARG(grid.y <= 65535, "stream_copies: rows of %d exceed the grid", width);
#define FRB_COPIES(MOST) \
    launch_dependent(x_out ? copies_kernel<OutT, MOST, true> : copies_kernel<OutT, MOST, false>, grid, dim3(COPIES_BLOCK), 0, stream, p)
    FRB_DISPATCH_DTYPE(out_dtype, OutT, {
        if (!by_four) {
            const size_t smem = ((size_t)streams * streams + 3 * streams + (size_t)streams * COPIES_BLOCK) * sizeof(float);
            auto kernel = copies_any_kernel<OutT>;
            if (smem > 40 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            launch_dependent(kernel, grid, dim3(COPIES_BLOCK), smem, stream, p);
        } else if (streams <= 2) FRB_COPIES(2);
        else if (streams <= 4) FRB_COPIES(4);
        else FRB_COPIES(8);
    });
#undef FRB_COPIES
    FRB_RETURN_LAUNCH("stream_copies");
}
