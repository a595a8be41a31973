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

__device__ __forceinline__ float rb_relu2(float z) { const float r = fmaxf(z, 0.0f); return r * r; }
__device__ __forceinline__ float rb_gelu(float z) { return 0.5f * z * (1.0f + erff(z * 0.70710678118654752f)); }
// 0.5 (1 + tanh u) = 1 / (1 + exp(-2u)), u = sqrt(2/pi) (z + 0.044715 z^3)
__device__ __forceinline__ float rb_gelu_tanh(float z) { return z / (1.0f + expf(-1.5957691216057308f * (z + 0.044715f * z * z * z))); }

// v[i] <- f(v[i]) * fac[i].  The choice of f lies outside the loops, so that the N results are independent chains.
template <int N>
__device__ __forceinline__ void rb_act_finish(int kind, float (&v)[N], const float (&fac)[N]) {
    if (kind == 1) {
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] = rb_relu2(v[i]) * fac[i];
    } else if (kind == 2) {
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] = rb_gelu(v[i]) * fac[i];
    } else if (kind == 3) {
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] = rb_gelu_tanh(v[i]) * fac[i];
    } else {
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] *= fac[i];
    }
    // (a factor of zero leaves a zero whatever stands before it)
#pragma unroll
    for (int i = 0; i < N; ++i) if (fac[i] == 0.0f) v[i] = 0.0f;
}

// The pointwise middle of a gated pair (two products side by side, gate and up):
//
//   kind 0   silu(g) * u              silu(z) = z sigmoid(z)
//   kind 1   gelu(g) * u              the tanh form
//   kind 2   g' sigmoid(1.702 g') (u' + 1),   g' = min(g, limit),  u' = u cut to [-limit, limit]
//
// then times the token's factor for the column's block: `gates` rows of gate_ld numbers (null: none), blocks of `ff` columns;
// all columns behind the first `blocks` blocks share the factor with index `blocks` and take `tail_limit` for their limit
// (a shared expert of a size and a constant of its own).  `bias` [2F] (null: none) joins g and u first.  `up_row`: how many
// weight rows lie between a column's gate row and its up row.
struct RbGlu {
    const float* bias;
    const float* gates;
    int kind, ff, blocks, F, gate_ld, up_row;
    float limit, tail_limit;
};

__device__ __forceinline__ float rb_glu_value(const RbGlu& gl, float g, float u, int block) {
    if (gl.kind == 2) {
        const float lim = block < gl.blocks ? gl.limit : gl.tail_limit;
        g = fminf(g, lim);
        u = fminf(fmaxf(u, -lim), lim);
        return g / (1.0f + expf(-1.702f * g)) * (u + 1.0f);
    }
    // tanh-gelu: 0.5 (1 + tanh(u)) = 1 / (1 + exp(-2u)), u = sqrt(2/pi) (g + 0.044715 g^3) - one exponential, as silu
    return g / (1.0f + expf(gl.kind == 1 ? -1.5957691216057308f * (g + 0.044715f * g * g * g) : -g)) * u;
}
__device__ __forceinline__ int rb_glu_block(const RbGlu& gl, int col) { const int e = col / gl.ff; return e < gl.blocks ? e : gl.blocks; }
__device__ __forceinline__ float rb_glu(const RbGlu& gl, float g, float u, int col, int tok) {
    if (gl.bias) { g += gl.bias[col]; u += gl.bias[gl.F + col]; }
    if (!gl.gates && gl.kind != 2) return rb_glu_value(gl, g, u, 0);
    const int b = rb_glu_block(gl, col);
    float v = rb_glu_value(gl, g, u, b);
    if (gl.gates) v *= gl.gates[(size_t)tok * gl.gate_ld + b];
    return v;
}

// N neighbouring columns of one token, for results that are rounded to bfloat16 on the way out: g <- f(g, u) * factor.  Blocks are
// looked up once where the columns share one, and the choice of f lies outside the loops, so that the N results are independent
// chains; kind 2 takes the fast exponential and division.  (Columns at or beyond F are computed from the last one's factors
// and not stored by the caller.)
template <int N>
__device__ __forceinline__ void rb_glu_cols(const RbGlu& gl, float (&g)[N], float (&u)[N], int col0, int tok, int F) {
    if (gl.bias) {
#pragma unroll
        for (int i = 0; i < N; ++i) { const int c = min(col0 + i, F - 1); g[i] += gl.bias[c]; u[i] += gl.bias[gl.F + c]; }
    }
    float w[N], lim[N];
    if (gl.gates || gl.kind == 2) {
        const float* row = gl.gates ? gl.gates + (size_t)tok * gl.gate_ld : nullptr;
        const int first = rb_glu_block(gl, min(col0, F - 1)), last = rb_glu_block(gl, min(col0 + N, F) - 1);
        if (first == last) {
            const float w0 = row ? row[first] : 1.0f, l0 = first < gl.blocks ? gl.limit : gl.tail_limit;
#pragma unroll
            for (int i = 0; i < N; ++i) { w[i] = w0; lim[i] = l0; }
        } else {
#pragma unroll
            for (int i = 0; i < N; ++i) {
                const int b = rb_glu_block(gl, min(col0 + i, F - 1));
                w[i] = row ? row[b] : 1.0f;
                lim[i] = b < gl.blocks ? gl.limit : gl.tail_limit;
            }
        }
    } else {
#pragma unroll
        for (int i = 0; i < N; ++i) w[i] = 1.0f;
    }
    if (gl.kind == 2) {
#pragma unroll
        for (int i = 0; i < N; ++i) {
            const float a = fminf(g[i], lim[i]), b = fminf(fmaxf(u[i], -lim[i]), lim[i]);
            g[i] = __fdividef(a, 1.0f + __expf(-1.702f * a)) * (b + 1.0f) * w[i];
        }
    } else if (gl.kind == 1) {
#pragma unroll
        for (int i = 0; i < N; ++i) g[i] = rb_gelu_tanh(g[i]) * u[i] * w[i];
    } else {
#pragma unroll
        for (int i = 0; i < N; ++i) g[i] = g[i] / (1.0f + expf(-g[i])) * u[i] * w[i];
    }
}

// The arguments as the entry points take them, checked: F columns (blocks 0: as many blocks of ff as there are columns for).
static inline int rb_glu_make(RbGlu* g, const float* bias, int kind, const float* gates, int gate_ld, int ff, int blocks, float limit,
                              float tail_limit, int up_row, int F) {
    if (kind < 0 || kind > 2) RB_REFUSE("gated pair: activation %d (0..2)", kind);
    if (ff <= 0) { ff = F; blocks = 1; }
    if (blocks <= 0) {
        if (F % ff) RB_REFUSE("gated pair: %d columns in blocks of %d", F, ff);
        blocks = F / ff;
    }
    const bool tail = (long long)blocks * ff < F;
    if ((long long)blocks * ff > F || (gates && gate_ld < blocks + (tail ? 1 : 0)))
        RB_REFUSE("gated pair: %d columns as %d blocks of %d with rows of %d factors", F, blocks, ff, gate_ld);
    if (kind == 2 && (!(limit > 0.0f) || (tail && !(tail_limit > 0.0f)))) RB_REFUSE("gated pair: limits %f and %f", limit, tail_limit);
    if (up_row < 0 || (up_row > 0 && up_row < F)) RB_REFUSE("gated pair: up rows %d behind the gate rows of %d columns", up_row, F);
    *g = RbGlu{bias, gates, kind, ff, blocks, F, gates ? gate_ld : 0, up_row ? up_row : F, limit, tail_limit};
    return 0;
}

// The index of a column's factor in its token's row of gates.
__device__ __forceinline__ int rb_act_block(const RbAct& a, int col) { const int e = col / a.ff; return e < a.blocks ? e : a.blocks; }

// N neighbouring columns of one token (columns at or beyond F are computed from the last one's factors and not stored by
// the caller): all loads first, then the arithmetic.
template <int N>
__device__ __forceinline__ void rb_act_cols(const RbAct& a, float (&v)[N], int col0, int tok, int F) {
    float fac[N];
#pragma unroll
    for (int i = 0; i < N; ++i) fac[i] = a.scale;
    if (a.gates) {
        const float* row = a.gates + (size_t)tok * a.gate_ld;
        const int first = rb_act_block(a, col0), last = rb_act_block(a, min(col0 + N, F) - 1);
        if (first == last) {
            const float g = row[first];
#pragma unroll
            for (int i = 0; i < N; ++i) fac[i] *= g;
        } else {
            float g[N];
#pragma unroll
            for (int i = 0; i < N; ++i) g[i] = row[rb_act_block(a, min(col0 + i, F - 1))];
#pragma unroll
            for (int i = 0; i < N; ++i) fac[i] *= g[i];
        }
    }
    if (a.mul) {
        const size_t at = (size_t)a.mul_row[tok] * a.mul_ld + col0;
        if (!a.mul_f32 && N % 8 == 0 && col0 + N <= F && (((uintptr_t)((const bf16*)a.mul + at)) & 15) == 0) {
            uint4 raw[N / 8 > 0 ? N / 8 : 1];
#pragma unroll
            for (int i = 0; i < N / 8; ++i) raw[i] = reinterpret_cast<const uint4*>((const bf16*)a.mul + at)[i];
#pragma unroll
            for (int i = 0; i < N / 8; ++i) {
                const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&raw[i]);
#pragma unroll
                for (int k = 0; k < 4; ++k) { const float2 f = __bfloat1622float2(h2[k]); fac[8 * i + 2 * k] *= f.x; fac[8 * i + 2 * k + 1] *= f.y; }
            }
        } else {
            float g[N];
#pragma unroll
            for (int i = 0; i < N; ++i) {
                const size_t p = at + (size_t)(min(col0 + i, F - 1) - col0);
                g[i] = a.mul_f32 ? ((const float*)a.mul)[p] : __bfloat162float(((const bf16*)a.mul)[p]);
            }
#pragma unroll
            for (int i = 0; i < N; ++i) fac[i] *= g[i];
        }
    }
    rb_act_finish<N>(a.kind, v, fac);
}

// One column of N neighbouring tokens, of which the first n exist.
template <int N>
__device__ __forceinline__ void rb_act_toks(const RbAct& a, float (&v)[N], int col, int tok0, int n) {
    float fac[N];
#pragma unroll
    for (int i = 0; i < N; ++i) fac[i] = a.scale;
    if (a.gates) {
        const float* row = a.gates + (size_t)tok0 * a.gate_ld + rb_act_block(a, col);
        float g[N];
#pragma unroll
        for (int i = 0; i < N; ++i) g[i] = row[(size_t)min(i, n - 1) * a.gate_ld];
#pragma unroll
        for (int i = 0; i < N; ++i) fac[i] *= g[i];
    }
    if (a.mul) {
        int r[N];
        float g[N];
#pragma unroll
        for (int i = 0; i < N; ++i) r[i] = a.mul_row[tok0 + min(i, n - 1)];
#pragma unroll
        for (int i = 0; i < N; ++i) {
            const size_t p = (size_t)r[i] * a.mul_ld + col;
            g[i] = a.mul_f32 ? ((const float*)a.mul)[p] : __bfloat162float(((const bf16*)a.mul)[p]);
        }
#pragma unroll
        for (int i = 0; i < N; ++i) fac[i] *= g[i];
    }
    rb_act_finish<N>(a.kind, v, fac);
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
