// A feed-forward's activation that looks at its whole row: out = a N(z) + b N(z^2) + c N(z^3) + e, powers element by element,
// N(v) = v / sqrt(mean(v^2) + eps) over the row, (a, b, c, e) four learned numbers.  One block per row; the three mean squares
// are means of z^2, z^4 and z^6, so one pass over the row makes all of them, and the row stays in registers for the second.
// Float32 throughout; the result is rounded once.
#include "common.cuh"

template <int BLOCK>
__device__ __forceinline__ void block_sum_three(float& a, float& b, float& c, float (*scratch)[32]) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    a = warp_sum(a);
    b = warp_sum(b);
    c = warp_sum(c);
    if (lane == 0) { scratch[0][warp] = a; scratch[1][warp] = b; scratch[2][warp] = c; }
    __syncthreads();
    // every warp adds the warps' sums for itself, in the same order
    a = warp_sum(lane < BLOCK / 32 ? scratch[0][lane] : 0.f);
    b = warp_sum(lane < BLOCK / 32 ? scratch[1][lane] : 0.f);
    c = warp_sum(lane < BLOCK / 32 ? scratch[2][lane] : 0.f);
}

struct PolyNorm {
    float c1, c2, c3, c0;
    __device__ __forceinline__ PolyNorm(const float* act, float ss2, float ss4, float ss6, float width, float eps) {
        c1 = act[0] / sqrtf(ss2 / width + eps);
        c2 = act[1] / sqrtf(ss4 / width + eps);
        c3 = act[2] / sqrtf(ss6 / width + eps);
        c0 = act[3];
    }
    __device__ __forceinline__ float operator()(float z) const { return fmaf(z, fmaf(z, fmaf(z, c3, c2), c1), c0); }
};

__device__ __forceinline__ void add_powers(float z, float& ss2, float& ss4, float& ss6) {
    const float z2 = z * z, z4 = z2 * z2;
    ss2 += z2;
    ss4 += z4;
    ss6 = fmaf(z4, z2, ss6);
}

// GROUPS: groups of four elements that a thread keeps.
template <typename OutT, int BLOCK, int GROUPS>
__global__ void __launch_bounds__(BLOCK) poly_norm_kernel(const float* __restrict__ in, const float* __restrict__ act,
                                                          OutT* __restrict__ out, int width, float eps) {
    __shared__ float scratch[3][32];
    after_previous_kernel();
    const float* row = in + (size_t)blockIdx.x * width;
    float4 z[GROUPS];
#pragma unroll
    for (int u = 0; u < GROUPS; ++u) {
        const int i = 4 * (u * BLOCK + threadIdx.x);
        z[u] = i < width ? *reinterpret_cast<const float4*>(row + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    float ss2 = 0.f, ss4 = 0.f, ss6 = 0.f;
#pragma unroll
    for (int u = 0; u < GROUPS; ++u) {
        add_powers(z[u].x, ss2, ss4, ss6);
        add_powers(z[u].y, ss2, ss4, ss6);
        add_powers(z[u].z, ss2, ss4, ss6);
        add_powers(z[u].w, ss2, ss4, ss6);
    }
    block_sum_three<BLOCK>(ss2, ss4, ss6, scratch);
    const PolyNorm f(act, ss2, ss4, ss6, (float)width, eps);
    OutT* dst = out + (size_t)blockIdx.x * width;
#pragma unroll
    for (int u = 0; u < GROUPS; ++u) {
        const int i = 4 * (u * BLOCK + threadIdx.x);
        if (i < width) {
            const float4 y = make_float4(f(z[u].x), f(z[u].y), f(z[u].z), f(z[u].w));
            if constexpr (sizeof(OutT) == 4) {
                *reinterpret_cast<float4*>(dst + i) = y;
            } else {
                const __nv_bfloat162 lo = __floats2bfloat162_rn(y.x, y.y), hi = __floats2bfloat162_rn(y.z, y.w);
                uint2 raw;
                raw.x = *reinterpret_cast<const unsigned int*>(&lo);
                raw.y = *reinterpret_cast<const unsigned int*>(&hi);
                *reinterpret_cast<uint2*>(dst + i) = raw;
            }
        }
    }
}

// Any width: the row is read twice.
template <typename OutT>
__global__ void __launch_bounds__(256) poly_norm_any_kernel(const float* __restrict__ in, const float* __restrict__ act,
                                                            OutT* __restrict__ out, int width, float eps) {
    __shared__ float scratch[3][32];
    after_previous_kernel();
    const float* row = in + (size_t)blockIdx.x * width;
    float ss2 = 0.f, ss4 = 0.f, ss6 = 0.f;
    for (int i = threadIdx.x; i < width; i += 256) add_powers(row[i], ss2, ss4, ss6);
    block_sum_three<256>(ss2, ss4, ss6, scratch);
    const PolyNorm f(act, ss2, ss4, ss6, (float)width, eps);
    for (int i = threadIdx.x; i < width; i += 256) out[(size_t)blockIdx.x * width + i] = from_f32<OutT>(f(row[i]));
}

#define POLY_FEW_ROWS 64       // up to this many rows a row's latency is the step's: blocks of 1024 threads

FRB_API int frb_poly_norm(const float* in, const float* act, void* out, int out_dtype, int num_rows, int width, float eps,
                          cudaStream_t stream) {
    if (num_rows == 0) return 0;
    const bool by_four = width % 4 == 0 && ((uintptr_t)in & 15) == 0 && ((uintptr_t)out & 15) == 0;
    const int few = num_rows <= POLY_FEW_ROWS;
    const int per_block = few ? 4096 : 1024;                    // elements of a group of four per thread
    const int groups = (width + per_block - 1) / per_block;
#define FRB_POLY(BLOCK, GROUPS) \
    launch_dependent(poly_norm_kernel<OutT, BLOCK, GROUPS>, dim3(num_rows), dim3(BLOCK), 0, stream, in, act, (OutT*)out, width, eps)
    FRB_DISPATCH_DTYPE(out_dtype, OutT, {
        if (!by_four || width > 32768) launch_dependent(poly_norm_any_kernel<OutT>, dim3(num_rows), dim3(256), 0, stream, in, act, (OutT*)out, width, eps);
        else if (few) {
            if (groups <= 1) FRB_POLY(1024, 1); else if (groups <= 2) FRB_POLY(1024, 2); else if (groups <= 4) FRB_POLY(1024, 4); else FRB_POLY(1024, 8);
        } else {
            if (groups <= 2) FRB_POLY(256, 2); else if (groups <= 4) FRB_POLY(256, 4); else if (groups <= 8) FRB_POLY(256, 8);
            else if (groups <= 16) FRB_POLY(1024, 4); else FRB_POLY(1024, 8);
        }
    });
#undef FRB_POLY
    FRB_RETURN_LAUNCH("poly_norm");
}
