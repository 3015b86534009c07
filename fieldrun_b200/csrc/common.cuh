// Shared helpers of the sm_100a kernels: element types, reductions with a fixed order,
// the error string that the C entry points leave for the Python side.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <cstdlib>
#include <stdint.h>
#include <stdio.h>

#define FRB_API extern "C" __attribute__((visibility("default")))

typedef __nv_bfloat16 bf16;

// Element type codes used by every entry point.
enum FrbDtype { FRB_F32 = 0, FRB_BF16 = 1 };

// Tokens per cache page; must equal PAGE_TOKENS of the Python cache.
#define FRB_PAGE 64

void frb_set_error(const char* fmt, ...);

#define FRB_CHECK_ARG(cond, ...)            \
    do {                                    \
        if (!(cond)) {                      \
            frb_set_error(__VA_ARGS__);     \
            return -1;                      \
        }                                   \
    } while (0)

#define FRB_RETURN_LAUNCH(name)                                                   \
    do {                                                                          \
        cudaError_t frb_e_ = cudaGetLastError();                                  \
        if (frb_e_ != cudaSuccess) {                                              \
            frb_set_error("%s: launch failed: %s", name, cudaGetErrorString(frb_e_)); \
            return (int)frb_e_;                                                   \
        }                                                                         \
        return 0;                                                                 \
    } while (0)

// Programmatic dependent launch.  A kernel started with launch_dependent() may begin while the kernel before
// it in the stream still runs; it calls after_previous_kernel() before it reads or writes anything, which
// first lets the kernel after it begin in the same way and then waits until the kernel before it has ended
// and its writes are visible.  What the launch hides is the time between one kernel's last block and the next
// kernel's first instruction, which is most of the cost of the small kernels of a decode step.  In a kernel
// that was started in the ordinary way both instructions do nothing.
//
// A kernel may also do work that does not depend on the kernel before it (loading weights) ahead of
// wait_for_previous_kernel().  If it reads, ahead of the wait, what a kernel two or more places before it in the
// stream wrote, then the kernel directly before it must call let_next_kernel_start() only after its own wait.
__device__ __forceinline__ void let_next_kernel_start() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void wait_for_previous_kernel() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void after_previous_kernel() {
    let_next_kernel_start();
    wait_for_previous_kernel();
}

// The largest grid that is started early: the number of SMs, or FIELDRUN_B200_PDL from the environment
// (0 starts every kernel in the ordinary way).  Blocks that start early settle on whichever SMs have room at
// that moment; a kernel of many blocks that is bound by memory bandwidth then runs from an uneven placement
// and loses more than the early start gains, so only the small kernels are started early.
inline long frb_dependent_launch_blocks() {
    static const long most = [] {
        const char* v = getenv("FIELDRUN_B200_PDL");
        if (v && v[0]) return atol(v);
        int device = 0, sms = 0;
        cudaGetDevice(&device);
        cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, device);
        return (long)sms;
    }();
    return most;
}

// Starts `kernel`, which orders itself behind the kernel before it with the instructions above, early if its grid
// has at most `per_sm` blocks for every SM (all of them must be able to be resident at once).
template <typename... Params, typename... Args>
inline void launch_dependent_resident(int per_sm, void (*kernel)(Params...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                                      Args... args) {
    cudaLaunchConfig_t config = {};
    config.gridDim = grid;
    config.blockDim = block;
    config.dynamicSmemBytes = smem;
    config.stream = stream;
    cudaLaunchAttribute attribute[1];
    attribute[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attribute[0].val.programmaticStreamSerializationAllowed = 1;
    config.attrs = attribute;
    config.numAttrs = (long)grid.x * grid.y * grid.z <= per_sm * frb_dependent_launch_blocks() ? 1 : 0;
    cudaLaunchKernelEx(&config, kernel, Params(args)...);
}

// Starts `kernel`, whose first statement is after_previous_kernel(), early if its grid has at most a block per SM.
template <typename... Params, typename... Args>
inline void launch_dependent(void (*kernel)(Params...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream, Args... args) {
    launch_dependent_resident(1, kernel, grid, block, smem, stream, args...);
}

// The first key that the query at `pos` may see: with a window the last `window` keys, with chunks the keys of its own
// chunk of `chunk` positions (chunks counted from position 0); 0 switches either off.
__device__ __forceinline__ int first_visible_key(int pos, int window, int chunk) {
    int lo = window > 0 ? max(0, pos - window + 1) : 0;
    if (chunk > 0) lo = max(lo, pos / chunk * chunk);
    return lo;
}

// A query whose sequence keeps its first `keep_first` tokens visible beside the window looks at two runs of pages: the
// pages of those tokens, as far as they lie before `first_page`, then the pages from `first_page` on.  kept_runs() is the
// number of units (pages, or any other size) of the first run, run_at() the unit that comes n-th; key_visible() what holds
// inside them.
__device__ __forceinline__ int kept_runs(int keep_first, int unit, int first) { return min((keep_first + unit - 1) / unit, first); }
__device__ __forceinline__ int run_at(int n, int kept, int first) { return n < kept ? n : first + n - kept; }
__device__ __forceinline__ bool key_visible(int key, int lo, int hi, int keep_first) {
    return (key >= lo || key < keep_first) && key <= hi;
}

// A capped attention score for kernels that keep scores as powers of two: raw * scale becomes cap * tanh(raw * scale / cap),
// returned times log2(e).  cap_scale = scale / cap, cap2 = cap * log2(e).  tanh(x) = 1 - 2 / (exp(2x) + 1) with the
// hardware's exponential and reciprocal (errors of a few 1e-7 of the cap: these kernels round the weights to bfloat16).
__device__ __forceinline__ float capped_score2(float raw, float cap_scale, float cap2) {
    const float x = fminf(raw * cap_scale, 40.f);
    const float e = exp2f(x * 2.8853900817779268f);
    return cap2 * (1.0f - __fdividef(2.0f, e + 1.0f));
}

template <typename T> __device__ __forceinline__ float to_f32(T v);
template <> __device__ __forceinline__ float to_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f32<bf16>(bf16 v) { return __bfloat162float(v); }

template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// Sum over a block of BLOCK threads; every thread gets the result.  The order of additions depends on
// BLOCK only, so a row's sum is the same whatever else the launch holds.  `scratch` holds 32 floats.
// One warp adds the warps' sums: with every thread reading all of them, a block of 1024 threads made a thousand
// shared-memory loads per call, half a microsecond of a decode step's norm.
template <int BLOCK>
__device__ __forceinline__ float block_sum(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    v = warp_sum(v);
    __syncthreads();                      // scratch may still be read from an earlier call
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    if (warp == 0) {
        const float total = warp_sum(lane < BLOCK / 32 ? scratch[lane] : 0.f);
        if (lane == 0) scratch[0] = total;
    }
    __syncthreads();
    return scratch[0];
}

// Two sums at once (the squares of a token's query and key rows).  `scratch` holds 64 floats.
template <int BLOCK>
__device__ __forceinline__ void block_sum_pair(float& a, float& b, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    a = warp_sum(a);
    b = warp_sum(b);
    __syncthreads();                      // scratch may still be read from an earlier call
    if (lane == 0) { scratch[warp] = a; scratch[32 + warp] = b; }
    __syncthreads();
    if (warp == 0) {
        const float total_a = warp_sum(lane < BLOCK / 32 ? scratch[lane] : 0.f);
        const float total_b = warp_sum(lane < BLOCK / 32 ? scratch[32 + lane] : 0.f);
        if (lane == 0) { scratch[0] = total_a; scratch[32] = total_b; }
    }
    __syncthreads();
    a = scratch[0];
    b = scratch[32];
}

// The gate of a feed-forward unit with two products in: silu(gate) * up, or, with a positive `limit`, the clamped form
// g = min(gate, limit), u = clamp(up, -limit, limit), g * sigmoid(1.702 g) * (u + 1).
#define FRB_CLAMPED_GATE_SLOPE 1.702f
__device__ __forceinline__ float paired_gate(float gate, float up, float limit) {
    if (limit > 0.f) {
        const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
        return g / (1.0f + expf(-FRB_CLAMPED_GATE_SLOPE * g)) * (u + 1.0f);
    }
    return gate / (1.0f + expf(-gate)) * up;
}

// Calls `body` with a value of the element type that `code` names.
#define FRB_DISPATCH_DTYPE(code, T, ...)                          \
    do {                                                          \
        if ((code) == FRB_F32) { typedef float T; __VA_ARGS__; }  \
        else { typedef bf16 T; __VA_ARGS__; }                     \
    } while (0)
