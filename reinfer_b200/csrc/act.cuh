// The pointwise end of a product that makes a feed-forward's inner rows from ONE matrix (no gate matrix beside it):
//
//   out[t, c] = f(z[t, c]) * scale * gates[t, block of c] * mul[mul_row[t], c]
//
// f: 0 nothing, 1 squared relu, 2 gelu (the error function's), 3 the tanh form of gelu.  Every factor is optional (null;
// scale 1).  gates: float rows of `gate_ld` numbers, one factor per token and block of `ff` columns - an expert of a mixture
// whose experts' matrices were stacked - where all columns behind the first `blocks` blocks share the factor with index
// `blocks` (a shared expert of a size of its own); a factor of zero leaves an exact zero.  mul: rows of bfloat16 or float
// numbers picked per token.  32-bit arithmetic.
#pragma once
#include "common.cuh"

struct RbAct {
    int kind;                    // -1: the product takes no part in this
    float scale;
    const float* gates;
    int gate_ld, ff, blocks;
    const void* mul;
    int mul_f32;
    long long mul_ld;
    const int* mul_row;
};

__device__ __forceinline__ float rb_act_f(float z, int kind) {
    if (kind == 1) { const float r = fmaxf(z, 0.0f); return r * r; }
    if (kind == 2) return 0.5f * z * (1.0f + erff(z * 0.70710678118654752f));
    if (kind == 3) return z / (1.0f + expf(-1.5957691216057308f * (z + 0.044715f * z * z * z)));   // 0.5 (1 + tanh u) = 1 / (1 + exp(-2u))
    return z;
}

__device__ __forceinline__ float rb_act(const RbAct& a, float z, int col, int tok) {
    float f = a.scale;
    if (a.gates) {
        const int e = col / a.ff;
        f *= a.gates[(size_t)tok * a.gate_ld + (e < a.blocks ? e : a.blocks)];
        if (f == 0.0f) return 0.0f;
    }
    if (a.mul) {
        const size_t at = (size_t)a.mul_row[tok] * a.mul_ld + col;
        f *= a.mul_f32 ? ((const float*)a.mul)[at] : __bfloat162float(((const bf16*)a.mul)[at]);
    }
    return rb_act_f(z, a.kind) * f;
}

// The arguments as the entry points take them, checked: F columns.
static inline int rb_act_make(RbAct* a, int kind, float scale, const float* gates, int gate_ld, int ff, int blocks, const void* mul,
                              int mul_dtype, long long mul_ld, const int* mul_row, int F) {
    if (kind < 0 || kind > 3) RB_REFUSE("activation %d (0..3)", kind);
    if (gates && (ff <= 0 || blocks < 0 || (long long)blocks * ff > F || gate_ld < blocks + ((long long)blocks * ff < F ? 1 : 0)))
        RB_REFUSE("activation: %d columns as %d blocks of %d with rows of %d factors", F, blocks, ff, gate_ld);
    if (mul && (!mul_row || (mul_dtype != RB_F32 && mul_dtype != RB_BF16) || mul_ld < F)) RB_REFUSE("activation: rows to multiply with, of float or bfloat16, need the tokens' indices");
    *a = RbAct{kind, scale, gates, gates ? gate_ld : 0, gates ? ff : 1, gates ? blocks : 0, mul, mul_dtype == RB_F32, mul_ld, mul_row};
    return 0;
}
