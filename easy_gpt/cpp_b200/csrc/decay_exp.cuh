// exp(x) for x <= 0, for the decay factors of recurrent states.  A state that decays slowly is multiplied by thousands of
// such factors in a row, so an error with a sign of its own would add up over a long sequence where errors of either sign
// do not (measured on a sequence of 1,100 tokens: the logits were 4e-5 of their spread away from a float64 computation
// with expf, 1e-5 with factors rounded to nearest in all but rare cases).
//
// The mathematics: x = k ln 2 + r with an integer k and |r| <= ln 2 / 2, e^x = 2^k e^r, and e^r by its Taylor series
//   e^r = 1 + (r + r^2 (1/2! + r/3! + r^2/4! + r^3/5! + r^4/6! + r^5/7!)),
// whose remainder is below (ln 2 / 2)^8 / 8! < 5.3e-9, a twentieth of a unit in the last place.  k ln 2 is taken off in
// two pieces: the first, 11357/16384, has 14 bits, so that its product with k (at most 8 bits) is exact.  The addition
// of 1 is the only rounding that counts.  x_lo: what rounding x lost (a product's error), or 0.
#pragma once

__device__ __forceinline__ float decay_exp(float x, float x_lo = 0.0f) {
    constexpr double LN2 = 0.69314718055994530942, LN2_HEAD = 11357.0 / 16384.0;
    if (x < -104.0f) return 0.0f;                       // below half of the smallest float32
    const float k = rintf(x * (float)(1.0 / LN2));
    float r = fmaf(k, -(float)LN2_HEAD, x);
    r = fmaf(k, (float)(LN2_HEAD - LN2), r) + x_lo;
    float p = (float)(1.0 / 5040.0);
    p = fmaf(p, r, (float)(1.0 / 720.0));
    p = fmaf(p, r, (float)(1.0 / 120.0));
    p = fmaf(p, r, (float)(1.0 / 24.0));
    p = fmaf(p, r, (float)(1.0 / 6.0));
    p = fmaf(p, r, 0.5f);
    const float e = 1.0f + fmaf(r * r, p, r);
    const int ki = (int)k;                              // 2^k on the exponent; results below the normal range in two steps
    if (ki >= -125) return __int_as_float(__float_as_int(e) + (ki << 23));
    return __int_as_float(__float_as_int(e) + ((ki + 100) << 23)) * 7.888609052210118e-31f;      // 2^-100
}
