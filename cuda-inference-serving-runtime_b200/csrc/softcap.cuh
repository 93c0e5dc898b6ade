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
};
