// Scores of the tensor-core attention kernels: scale, softcap, exponent -- all in base 2, so that a probability is
// 2^t with t = log2(e) * score.
//
// A softcap C bounds |score| by C, so up to kFixedCap the exponentials need no running maximum: 2^t stays inside the
// fp32 (and bf16) exponent range against the fixed reference 0, and row sums and products against V with it.
#pragma once

#include "../ktk_umma.cuh"
#include "ktl_common.cuh"

namespace ktk {

constexpr float kLog2eF = 1.4426950408889634f;
constexpr float kFixedCap = 60.0f;      // e^60 ~ 1e26: sums over 2^24 keys and values up to 1e4 stay below 1e38

inline bool fixed_reference(const ktk_attn& a) { return a.softcap > 0.0f && a.softcap <= kFixedCap; }

// C log2(e) tanh(s f / C): 1 - 2 / (2^(2 x log2 e) + 1) has an absolute error of a few ulps of 1
struct CapCoef {
    float in, out;      // 2 log2(e) f / C, C log2(e)
    __device__ __forceinline__ void set(float factor, float cap) { in = 2.0f * kLog2eF * factor / cap; out = cap * kLog2eF; }
    __device__ __forceinline__ float operator()(float s) const {
        const float e = ex2(fminf(s * in, 126.0f));
        return out - __fdividef(2.0f * out, 1.0f + e);
    }
};

// The same on the FMA pipe for |s f / C| <= kPolyRange: tanh(x) = x P(x^2), P of degree 4 fitted for the smallest
// largest relative error on that range (Remez exchange): 1.0e-6.  Coefficients are scaled per row.
// Two fp32 operations per instruction.
__device__ __forceinline__ uint64_t pack2(float a, float b) {
    uint64_t r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ void unpack2(uint64_t v, float& a, float& b) {
    asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v));
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
    uint64_t r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}

constexpr float kPolyRange = 0.8f;
struct CapPoly {
    float c0, c1, c2, c3, c4, limit;
    __device__ __forceinline__ void set(float factor, float cap) {
        const float a = factor / cap, a2 = a * a, o = cap * kLog2eF;
        float w = o * a;
        c0 = 0.9999989867210388f * w; w *= a2;
        c1 = -0.3332537114620209f * w; w *= a2;
        c2 = 0.13230565190315247f * w; w *= a2;
        c3 = -0.04918014258146286f * w; w *= a2;
        c4 = 0.012100138701498508f * w;
        limit = kPolyRange / fmaxf(fabsf(a), 1e-30f);
    }
    __device__ __forceinline__ float operator()(float s) const {
        const float u = s * s;
        return s * fmaf(fmaf(fmaf(fmaf(c4, u, c3), u, c2), u, c1), u, c0);
    }
    __device__ __forceinline__ void two(float& a, float& b) const {
        const uint64_t s = pack2(a, b), u = mul2(s, s);
        uint64_t t = fma2(pack2(c4, c4), u, pack2(c3, c3));
        t = fma2(t, u, pack2(c2, c2));
        t = fma2(t, u, pack2(c1, c1));
        t = fma2(t, u, pack2(c0, c0));
        unpack2(mul2(s, t), a, b);
    }
};

}  // namespace ktk
