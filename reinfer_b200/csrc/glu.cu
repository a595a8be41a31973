// The pointwise middle of a gated feed-forward whose two first products come side by side, gu [T, gate: F | up: F]:
//
//   act[t, c] = f(gu[t, c] + b[c], gu[t, F + c] + b[F + c]) * gates[t, block of c]
//
// with the f's, blocks and limits of act.cuh (RbGlu).  The biases (float [2F]) and the gates (float rows: one factor per
// token and block of `ff` columns - an expert of a mixture whose experts' first products were stacked; zero where the
// expert was not chosen, and then nothing is read) are optional.
// The same for a feed-forward with one first matrix (rb_act_rows, see act.cuh).
// And the row vector that a last product's bias adds to every row of the float stream.  32-bit arithmetic, one
// rounding on the way out; a token's result depends on its own row only.
#include "act.cuh"

template <typename TI, typename TO>
__global__ void glu_act_kernel(const TI* __restrict__ gu, long long ld, RbGlu gl, TO* __restrict__ act, int T, int F) {
    pdl_trigger(); pdl_wait();
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= F) return;
    const float bg = gl.bias ? gl.bias[c] : 0.0f, bu = gl.bias ? gl.bias[F + c] : 0.0f;
    const int b = rb_glu_block(gl, c);
    for (int t = blockIdx.y; t < T; t += gridDim.y) {
        const float w = gl.gates ? gl.gates[(size_t)t * gl.gate_ld + b] : 1.0f;
        float v = 0.0f;
        if (w != 0.0f) {
            const TI* row = gu + (size_t)t * ld;
            v = rb_glu_value(gl, to_f32(row[c]) + bg, to_f32(row[F + c]) + bu, b) * w;
        }
        act[(size_t)t * F + c] = from_f32<TO>(v);
    }
}

// gu [T, 2F] rows with stride ld (float or bfloat16); act [T, F] contiguous.  The rest as in rb_glu_make.
extern "C" int rb_glu_act(const void* gu, long long ld, int in_dtype, const float* bias, int kind, const float* gates, int gate_ld,
                          int ff, int blocks, float limit, float tail_limit, void* act, int out_dtype, int T, int F, void* stream) {
    if (T <= 0 || F <= 0) return 0;
    RbGlu gl;
    if (rb_glu_make(&gl, bias, kind, gates, gate_ld, ff, blocks, limit, tail_limit, 0, F)) return -1;
    cudaStream_t s = (cudaStream_t)stream;
    dim3 grid(rb_ceil_div(F, 256), T < 65535 ? T : 65535);
#define GLU_GO(TI, TO) return rb_launch(glu_act_kernel<TI, TO>, grid, dim3(256), 0, s, (const TI*)gu, ld, gl, (TO*)act, T, F)
    if (in_dtype == RB_F32 && out_dtype == RB_F32) GLU_GO(float, float);
    if (in_dtype == RB_F32 && out_dtype == RB_BF16) GLU_GO(float, bf16);
    if (in_dtype == RB_BF16 && out_dtype == RB_BF16) GLU_GO(bf16, bf16);
#undef GLU_GO
    RB_REFUSE("glu_act: dtypes %d -> %d", in_dtype, out_dtype);
}

// x[t, :] += b for every row of the float stream; b float or bfloat16.
template <typename TB>
__global__ void add_row_vector_kernel(float* __restrict__ x, const TB* __restrict__ b, int T, int h) {
    pdl_trigger(); pdl_wait();
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= h) return;
    const float v = to_f32(b[c]);
    for (int t = blockIdx.y; t < T; t += gridDim.y) x[(size_t)t * h + c] += v;
}

extern "C" int rb_add_row_vector(float* x, const void* b, int b_dtype, int T, int h, void* stream) {
    if (T <= 0 || h <= 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    dim3 grid(rb_ceil_div(h, 256), T < 65535 ? T : 65535);
    if (b_dtype == RB_F32) return rb_launch(add_row_vector_kernel<float>, grid, dim3(256), 0, s, x, (const float*)b, T, h);
    if (b_dtype == RB_BF16) return rb_launch(add_row_vector_kernel<bf16>, grid, dim3(256), 0, s, x, (const bf16*)b, T, h);
    RB_REFUSE("add_row_vector: dtype %d", b_dtype);
}

// out[t, c] = f(u[t, c]) * scale * gate * row factor (act.cuh); u rows with stride ld (float or bfloat16), out [T, F] contiguous.
template <typename TI, typename TO>
__global__ void act_rows_kernel(const TI* __restrict__ u, long long ld, RbAct a, TO* __restrict__ out, int T, int F) {
    pdl_trigger(); pdl_wait();
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= F) return;
    for (int t = blockIdx.y; t < T; t += gridDim.y) {
        float v[1] = {to_f32(u[(size_t)t * ld + c])};
        rb_act_cols<1>(a, v, c, t, F);
        out[(size_t)t * F + c] = from_f32<TO>(v[0]);
    }
}

extern "C" int rb_act_rows(const void* u, long long ld, int in_dtype, void* out, int out_dtype, int T, int F, int kind, float scale,
                           const float* gates, int gate_ld, int ff, int blocks, const void* mul, int mul_dtype, long long mul_ld,
                           const int* mul_row, void* stream) {
    if (T <= 0 || F <= 0) return 0;
    RbAct a;
    if (rb_act_make(&a, kind, scale, gates, gate_ld, ff, blocks, mul, mul_dtype, mul_ld, mul_row, F)) return -1;
    cudaStream_t s = (cudaStream_t)stream;
    dim3 grid(rb_ceil_div(F, 256), T < 65535 ? T : 65535);
#define AR_GO(TI, TO) return rb_launch(act_rows_kernel<TI, TO>, grid, dim3(256), 0, s, (const TI*)u, ld, a, (TO*)out, T, F)
    if (in_dtype == RB_F32 && out_dtype == RB_F32) AR_GO(float, float);
    if (in_dtype == RB_F32 && out_dtype == RB_BF16) AR_GO(float, bf16);
    if (in_dtype == RB_BF16 && out_dtype == RB_BF16) AR_GO(bf16, bf16);
#undef AR_GO
    RB_REFUSE("act_rows: dtypes %d -> %d", in_dtype, out_dtype);
}
