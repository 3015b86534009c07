// What the tcgen05 prompt attention kernels share: arithmetic on pairs of float32, the hardware's exponential, capped scores.
#pragma once

#include "common.cuh"
#include "tcgen05.cuh"

#define AT_QUERIES 128
#define AT_RAISE 8.0f          // the running maximum follows a page's maximum only beyond this margin (in units of log2)

namespace frb_at {

// 2^x by the special-function unit (relative error about 2^-22; -inf and anything below -126 give 0)
__device__ __forceinline__ float exp2_fast(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// the largest of three (one instruction on this architecture)
__device__ __forceinline__ float max3(float a, float b, float c) {
    float d;
    asm("max.f32 %0, %1, %2, %3;" : "=f"(d) : "f"(a), "f"(b), "f"(c));
    return d;
}

// the hardware's instructions on two float32 values in one 64-bit register
__device__ __forceinline__ uint64_t pair_of(float lo, float hi) {
    uint64_t r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ void halves_of(uint64_t v, float& lo, float& hi) {
    asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
}
__device__ __forceinline__ uint64_t fma_pairs(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ uint64_t add_pairs(uint64_t a, uint64_t b) {
    uint64_t d;
    asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}


__device__ __forceinline__ uint64_t mul_pairs(uint64_t a, uint64_t b) {
    uint64_t d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}

// tanh(x) of a page's scores x = raw * cap_scale, in place.  Where no score of the warp's rows passes 0.4 of the cap: the
// Taylor series x (1 - x^2/3 + 2 x^4/15 - 17 x^6/315 + 62 x^8/2835 - 1382 x^10/155925), whose next term is below 1e-7 of x
// there, two scores at a time on the multiply-add pipe; else 1 - 2 / (exp(2x) + 1) with the hardware's exponential and
// reciprocal (two trips to the special-function unit a score, beside the softmax's own).
#define AT_SERIES_REACH 0.4f

template <int N>
__device__ __forceinline__ void cap_scores(uint32_t (&raw)[N][16], float cap_scale) {
    float top[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int c = 0; c < N; ++c)
#pragma unroll
        for (int i = 0; i < 16; i += 2)
            top[(i >> 1) & 3] = max3(top[(i >> 1) & 3], fabsf(__uint_as_float(raw[c][i])), fabsf(__uint_as_float(raw[c][i + 1])));
    const float most = fmaxf(fmaxf(top[0], top[1]), fmaxf(top[2], top[3])) * cap_scale;
    if (__all_sync(0xffffffffu, most <= AT_SERIES_REACH)) {
        const uint64_t scale = pair_of(cap_scale, cap_scale), one = pair_of(1.f, 1.f);
        const float k1 = -1.0f / 3.0f, k2 = 2.0f / 15.0f, k3 = -17.0f / 315.0f, k4 = 62.0f / 2835.0f, k5 = -1382.0f / 155925.0f;
        const uint64_t c1 = pair_of(k1, k1), c2 = pair_of(k2, k2), c3 = pair_of(k3, k3), c4 = pair_of(k4, k4), c5 = pair_of(k5, k5);
#pragma unroll
        for (int c = 0; c < N; ++c)
#pragma unroll
            for (int i = 0; i < 16; i += 2) {
                const uint64_t x = mul_pairs(pair_of(__uint_as_float(raw[c][i]), __uint_as_float(raw[c][i + 1])), scale);
                const uint64_t x2 = mul_pairs(x, x);
                uint64_t f = fma_pairs(x2, c5, c4);
                f = fma_pairs(x2, f, c3);
                f = fma_pairs(x2, f, c2);
                f = fma_pairs(x2, f, c1);
                f = fma_pairs(x2, f, one);
                float lo, hi;
                halves_of(mul_pairs(x, f), lo, hi);
                raw[c][i] = __float_as_uint(lo);
                raw[c][i + 1] = __float_as_uint(hi);
            }
    } else {
#pragma unroll
        for (int c = 0; c < N; ++c)
#pragma unroll
            for (int i = 0; i < 16; ++i) {
                const float e = exp2f(fminf(__uint_as_float(raw[c][i]) * cap_scale, 40.f) * 2.8853900817779268f);
                raw[c][i] = __float_as_uint(1.0f - __fdividef(2.0f, e + 1.0f));
            }
    }
}

}  // namespace frb_at
