// A soft cap on an attention score: c tanh(x / c) for c > 0 (inv_c = 1 / c), with tanh(y) = 1 - 2 / (e^(2y) + 1)
// from the fast exponential and division (absolute error about 1e-7 c).  The kernels that hold unscaled scores pass
// c = cap / scale, so that the scale they apply afterwards gives cap tanh(scale x / cap).  The cap is applied before
// the mask: a masked score stays the most negative number.
// Where every score of a block is far below the cap, |x| <= c / 2, tanh needs neither: x (1 + t (a1 + t (a2 + t (a3 + t a4))))
// with t = (x / c)^2 and the coefficients of the polynomial that interpolates tanh(y) / y in y^2 at the Chebyshev points of
// [0, 1/4] (relative error below 1.1e-7 in float32): a handful of multiply-adds where the exponential and the division take
// turns on one slow unit.
#pragma once

#define RI_SOFTCAP_SMALL 0.5f
#define RI_TANH_A1 -0.33333069f
#define RI_TANH_A2 0.13324751f
#define RI_TANH_A3 -0.052984238f
#define RI_TANH_A4 0.017131345f

__device__ __forceinline__ float ri_softcap(float x, float c, float inv_c) {
    float e;
    const float y = fminf(x * inv_c * 2.8853900817779268f, 64.0f);
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(y));
    return c * (1.0f - __fdividef(2.0f, e + 1.0f));
}
