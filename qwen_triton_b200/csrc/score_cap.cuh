// A cap on attention scores, s <- c tanh(s / c), for kernels that keep their scores unscaled (the score is the stored value times a
// positive `scale`, which is folded into the softmax's exponent later): stored <- (c / scale) tanh(stored * scale / c).
//
// Two forms, both float to rounding:
//   CAP_SMALL  |score / c| <= 1 for every score (known on the host, for instance where queries and keys have unit norm):
//              tanh(w) = w P(w^2), so stored <- stored P((stored * scale / c)^2) without a transcendental instruction.  P is the
//              polynomial of degree 6 through tanh(w) / w, fitted by least squares at 200 Chebyshev points of w^2 in [0, 1]
//              (relative error 5e-8 before rounding).
//   CAP_ANY    tanh(w) = 1 - 2 / (e^{2 w} + 1) with the hardware's ex2 and reciprocal; its absolute error is a few units of
//              2^-24, so the score's is that times c.
#pragma once

#include <stdint.h>

namespace qt {

constexpr int CAP_NONE = 0, CAP_SMALL = 1, CAP_ANY = 2;

struct ScoreCap {
    float in, out;          // scale / c, or for CAP_ANY 2 log2(e) scale / c; and c / scale
    template <int CAP> static __device__ __forceinline__ ScoreCap make(float softcap, float scale) {
        ScoreCap r;
        r.in = CAP == CAP_ANY ? 2.8853900817779268f * scale / softcap : scale / softcap;
        r.out = softcap / scale;
        return r;
    }
};

__device__ __forceinline__ float cap_polynomial(float x) {
    float p = fmaf(0.0010455536f, x, -0.00621706992f);
    p = fmaf(p, x, 0.0203055199f);
    p = fmaf(p, x, -0.0534651764f);
    p = fmaf(p, x, 0.133253977f);
    p = fmaf(p, x, -0.333328575f);
    return fmaf(p, x, 0.99999994f);
}

template <int CAP> __device__ __forceinline__ float capped(float s, const ScoreCap& c) {
    if (CAP == CAP_NONE) return s;
    if (CAP == CAP_SMALL) {
        const float w = s * c.in;
        return s * cap_polynomial(w * w);
    }
    float e, r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(s * c.in));
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(e + 1.f));
    return c.out * fmaf(-2.f, r, 1.f);
}

// Two scores at once (fma.rn.f32x2 and its like: every lane rounds as the one-wide form does).
__device__ __forceinline__ uint64_t cap_pair(float lo, float hi) {
    uint64_t d;
    asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
    return d;
}
__device__ __forceinline__ uint64_t cap_fma2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ uint64_t cap_mul2(uint64_t a, uint64_t b) {
    uint64_t d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ uint64_t capped_small2(uint64_t s, uint64_t in2) {
    const uint64_t w = cap_mul2(s, in2), x = cap_mul2(w, w);
    uint64_t p = cap_fma2(cap_pair(0.0010455536f, 0.0010455536f), x, cap_pair(-0.00621706992f, -0.00621706992f));
    p = cap_fma2(p, x, cap_pair(0.0203055199f, 0.0203055199f));
    p = cap_fma2(p, x, cap_pair(-0.0534651764f, -0.0534651764f));
    p = cap_fma2(p, x, cap_pair(0.133253977f, 0.133253977f));
    p = cap_fma2(p, x, cap_pair(-0.333328575f, -0.333328575f));
    p = cap_fma2(p, x, cap_pair(0.99999994f, 0.99999994f));
    return cap_mul2(s, p);
}

}  // namespace qt
