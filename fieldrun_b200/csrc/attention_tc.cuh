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

// Capped scores of a page, in place: cap2 * tanh(x) with x = raw * cap_scale (cap2 = cap * log2(e): the result is in units of
// log2).  Where no score of the warp's rows passes a fifth of the cap, or two fifths, the Taylor series of tanh serves,
//     x (1 - x^2/3 + 2 x^4/15 - 17 x^6/315 [+ 62 x^8/2835 - 1382 x^10/155925]),
// its next term below 1e-7 of x there, as a polynomial in raw^2 with the scales in its coefficients, two scores at a time on the
// multiply-add pipe; else 1 - 2 / (exp(2x) + 1) with the hardware's exponential and reciprocal (two trips to the special-function
// unit a score, beside the softmax's own).
template <int TERMS, int N>
__device__ __forceinline__ void cap_by_series(uint32_t (&raw)[N][16], float cap_scale, float cap2) {
    constexpr float series[6] = {1.0f, -1.0f / 3.0f, 2.0f / 15.0f, -17.0f / 315.0f, 62.0f / 2835.0f, -1382.0f / 155925.0f};
    uint64_t k[TERMS];
    float scale = cap_scale * cap2;
#pragma unroll
    for (int n = 0; n < TERMS; ++n) { k[n] = pair_of(series[n] * scale, series[n] * scale); scale *= cap_scale * cap_scale; }
#pragma unroll
    for (int c = 0; c < N; ++c) {
        // eight pairs a stage: a pair's own chain of dependent operations would wait for itself
        uint64_t x[8], x2[8], f[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            x[i] = pair_of(__uint_as_float(raw[c][2 * i]), __uint_as_float(raw[c][2 * i + 1]));
            x2[i] = mul_pairs(x[i], x[i]);
        }
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] = fma_pairs(x2[i], k[TERMS - 1], k[TERMS - 2]);
#pragma unroll
        for (int n = TERMS - 3; n >= 0; --n)
#pragma unroll
            for (int i = 0; i < 8; ++i) f[i] = fma_pairs(x2[i], f[i], k[n]);
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            float lo, hi;
            halves_of(mul_pairs(x[i], f[i]), lo, hi);
            raw[c][2 * i] = __float_as_uint(lo);
            raw[c][2 * i + 1] = __float_as_uint(hi);
        }
    }
}

template <int N>
__device__ __forceinline__ void cap_scores(uint32_t (&raw)[N][16], float cap_scale, float cap2) {
    float top[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int c = 0; c < N; ++c)
#pragma unroll
        for (int i = 0; i < 16; i += 2)
            top[(i >> 1) & 3] = max3(top[(i >> 1) & 3], fabsf(__uint_as_float(raw[c][i])), fabsf(__uint_as_float(raw[c][i + 1])));
    const float most = fmaxf(fmaxf(top[0], top[1]), fmaxf(top[2], top[3])) * cap_scale;
    if (__all_sync(0xffffffffu, most <= 0.2f)) {
        cap_by_series<4>(raw, cap_scale, cap2);
    } else if (__all_sync(0xffffffffu, most <= 0.4f)) {
        cap_by_series<6>(raw, cap_scale, cap2);
    } else {
#pragma unroll
        for (int c = 0; c < N; ++c)
#pragma unroll
            for (int i = 0; i < 16; ++i) raw[c][i] = __float_as_uint(capped_score2(__uint_as_float(raw[c][i]), cap_scale, cap2));
    }
}

}  // namespace frb_at
