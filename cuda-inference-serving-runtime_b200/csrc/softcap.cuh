// Scores bent smoothly into (-cap, cap) before the softmax: cap tanh(s / cap).
//
// The attention sources are compiled with -DSOFTCAP=1 for models whose scores are bent; without it the bend is the
// plain scaling it replaces and costs nothing.
#pragma once

#ifndef SOFTCAP
#define SOFTCAP 0
#endif

// In base-2 units, from the raw product of query and key: with z = score / cap, tanh z = 1 - 2 / (1 + e^(2z)), so
//   log2(e) cap tanh z = out - 2 out / (1 + 2^(in raw)),   in = 2 log2(e) scale / cap,   out = log2(e) cap.
// One exponential and one reciprocal; a product beyond the exponential's range gives +-out, as it should.
struct Bend {
    float in, out;
    __device__ __forceinline__ Bend(float scale, float cap)
        : in(2.f * 1.4426950408889634f * scale / cap), out(1.4426950408889634f * cap) {}
    __device__ __forceinline__ float operator()(float raw) const {
        float e, r;
        asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(raw * in));
        asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.f + e));
        return fmaf(-2.f * out, r, out);
    }
    // Four scores for one reciprocal: 1 / a = (1 / (a b c d)) (c d) b and so on.  The exponentials stop at 2^30, where tanh
    // is 1 to the last bit of a float, so the product of four stays finite.
    __device__ __forceinline__ void four(float& x0, float& x1, float& x2, float& x3) const {
        float a = x0, b = x1, c = x2, d = x3, r;
        asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(a) : "f"(fminf(a * in, 30.f)));
        asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(b) : "f"(fminf(b * in, 30.f)));
        asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(c) : "f"(fminf(c * in, 30.f)));
        asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(d) : "f"(fminf(d * in, 30.f)));
        a += 1.f; b += 1.f; c += 1.f; d += 1.f;
        const float ab = a * b, cd = c * d;
        asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(ab * cd));
        const float k = -2.f * out, rab = k * (r * cd), rcd = k * (r * ab);      // k / (a b), k / (c d)
        x0 = fmaf(rab, b, out);
        x1 = fmaf(rab, a, out);
        x2 = fmaf(rcd, d, out);
        x3 = fmaf(rcd, c, out);
    }
};
