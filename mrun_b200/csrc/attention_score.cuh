// What may be done to an attention score between the product and the softmax, and to a head's output
// behind it.  s = (q . k) * scale, then, in this order,
//   temperature   q at position p counts 1 + coef * ln(floor((p + 1) / every) + 1) times;
//   soft cap      s <- cap * tanh(s / cap);
//   bias          s <- s + bias[head][min(p - j, length - 1)], a table over distances in which the
//                 last entry stands for every longer one;
// and the head's output is multiplied, feature by feature, by sigmoid(gate) * out_scale on its way
// to memory.  Scores and gates are 32-bit.
//
// The tensor-core kernels carry this only where they are compiled with -DMRUN_SCORED=1.
#pragma once

#include "common.cuh"

// Passed by pointer through the C ABI (null: none of it); copied into the launch's arguments.
struct mrun_score_form {
    float cap;                // 0: no soft cap
    float temp_coef, temp_every;      // coef 0: no temperature
    float dot_bound;          // |q . k| never exceeds this (infinity where it is not known)
    const float* bias;        // [heads, bias_len] or null
    const void* gate;         // row t at gate + t * gate_stride (the activation type), a feature a column; or null
    long gate_stride;
    long out_stride;          // of the output's rows
    float out_scale;
    int bias_len;
};

namespace mrun {

__device__ __forceinline__ float query_temperature(const mrun_score_form& f, int pos) {
    if (f.temp_coef == 0.f) return 1.f;
    return 1.f + f.temp_coef * logf(floorf((float)(pos + 1) / f.temp_every) + 1.f);
}

// Scores in base-2 units from raw products, for one row (a query at one position of one head).
struct ScoreRow {
    float factor;             // of the raw product: into the tanh's argument times 2 log2(e), or into base-2 units
    float cap2;               // the cap in base-2 units, 0 without one
    bool small;               // |tanh's argument| <= 1/2 for every key: a polynomial serves
    const float* bias;        // the head's table, or null
    int bias_last;            // index of the entry for all longer distances
    float far_bias;           // that entry in base-2 units
};

__device__ __forceinline__ ScoreRow score_row(const mrun_score_form& f, float scale, int pos, int head) {
    constexpr float LOG2_E = 1.4426950408889634f;
    ScoreRow r;
    const float s = scale * query_temperature(f, pos < 0 ? 0 : pos);
    r.cap2 = f.cap * LOG2_E;
    r.small = f.cap > 0.f && f.dot_bound * fabsf(s) <= 0.5f * f.cap;
    r.factor = f.cap > 0.f ? (r.small ? s / f.cap : 2.f * LOG2_E * s / f.cap) : s * LOG2_E;
    r.bias = f.bias ? f.bias + (size_t)head * f.bias_len : nullptr;
    r.bias_last = f.bias_len - 1;
    r.far_bias = f.bias ? r.bias[r.bias_last] * LOG2_E : 0.f;
    return r;
}

// tanh for |y| <= 1/2 (a little more does no harm): the odd Taylor polynomial through y^11, whose first
// neglected term is y^13 * 21844 / 6081075, a relative 9e-7 at 1/2.
__device__ __forceinline__ float tanh_small(float y) {
    const float z = y * y;
    float p = -1382.f / 155925.f;
    p = fmaf(p, z, 62.f / 2835.f);
    p = fmaf(p, z, -17.f / 315.f);
    p = fmaf(p, z, 2.f / 15.f);
    p = fmaf(p, z, -1.f / 3.f);
    return fmaf(y * z, p, y);
}
__device__ __forceinline__ float2 tanh_small2(float2 y) {
    const float2 z = __fmul2_rn(y, y);
    auto both = [](float v) { return make_float2(v, v); };
    float2 p = both(-1382.f / 155925.f);
    p = __ffma2_rn(p, z, both(62.f / 2835.f));
    p = __ffma2_rn(p, z, both(-17.f / 315.f));
    p = __ffma2_rn(p, z, both(2.f / 15.f));
    p = __ffma2_rn(p, z, both(-1.f / 3.f));
    return __ffma2_rn(__fmul2_rn(y, z), p, y);
}

// The capped score without its bias, in base-2 units.  1 - 2 / (e^(2y) + 1) is tanh(y) with an absolute
// error of a few 2^-24, at either end of the range too (e^(2y) infinite gives 1, zero gives -1).
__device__ __forceinline__ float capped_score(const ScoreRow& r, float dot) {
    const float y = dot * r.factor;
    if (r.cap2 == 0.f) return y;
    if (r.small) return r.cap2 * tanh_small(y);
    float e, inv;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(y));
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(inv) : "f"(e + 1.f));
    return fmaf(-2.f * r.cap2, inv, r.cap2);
}

// The bias of a key `distance` positions back (negative: a key that the mask hides), in base-2 units.
__device__ __forceinline__ float distance_bias(const ScoreRow& r, int distance) {
    constexpr float LOG2_E = 1.4426950408889634f;
    if (!r.bias) return 0.f;
    return __ldg(r.bias + min(max(distance, 0), r.bias_last)) * LOG2_E;
}

// N consecutive features (an even number) of a bfloat16 output row, from feature `col` on.
template <int N>
__device__ __forceinline__ void gate_outputs(const mrun_score_form& f, size_t token, int col, float (&v)[N]) {
    if (f.gate) {
        const __nv_bfloat162* g = reinterpret_cast<const __nv_bfloat162*>((const __nv_bfloat16*)f.gate +
                                                                          token * f.gate_stride + col);
#pragma unroll
        for (int i = 0; i < N / 2; ++i) {
            const float2 x = __bfloat1622float2(g[i]);
            v[2 * i] *= f.out_scale / (1.f + __expf(-x.x));
            v[2 * i + 1] *= f.out_scale / (1.f + __expf(-x.y));
        }
    } else {
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] *= f.out_scale;
    }
}

__device__ __forceinline__ float gate_output(const mrun_score_form& f, size_t token, int col, float v) {
    if (!f.gate) return v * f.out_scale;
    const float g = __bfloat162float(((const __nv_bfloat16*)f.gate)[token * f.gate_stride + col]);
    return v * (f.out_scale / (1.f + __expf(-g)));
}

}  // namespace mrun
