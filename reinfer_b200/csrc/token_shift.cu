// Mixers whose projections read a blend of a token's row and the row of the token before it:
//
//   out[s][t, :] = h[t, :] + (h'[t, :] - h[t, :]) * mu[s, :]        s = 0 .. streams-1
//
// h' is the row of the request's previous token: the row above inside a portion, the request slot's row
// (state [slots, C], the activations' dtype) for a portion's first token - zeros for a request's first, since a slot is
// zeroed at admission.  The blend is 32-bit, rounded once.  The portion's last row becomes the slot's row: an entry of one
// token leaves it in the same thread that read the old one; for longer portions rb_keep_last_rows runs behind, after all
// reads.  A token's result depends on its own row and the one before it only.
//
// rb_keep_last_rows: state[entry_slot[e]] = rows[cu_q[e + 1] - 1] for every entry e of more than one token, rows of any
// plain type by their bytes.
#include "common.cuh"

#define TS_THREADS 128

// (h and state are not declared free of aliases: the row before a token is read through a pointer that may be either's, and the
// slot's row is written after that.)
template <typename TA, int VEC>
__global__ void __launch_bounds__(TS_THREADS)
token_shift_kernel(const TA* h, TA* state, const float* __restrict__ mu, TA* __restrict__ out,
                   const int* __restrict__ cu_q, const int* __restrict__ tok_entry, const int* __restrict__ entry_slot,
                   int T, int C, int streams) {
    pdl_trigger();
    const int c = (blockIdx.y * TS_THREADS + threadIdx.x) * VEC;
    const int t = blockIdx.x;
    const int e = tok_entry[t];
    const int first = cu_q[e], n = cu_q[e + 1] - first;
    TA* slot_row = state + (size_t)entry_slot[e] * C;
    pdl_wait();
    if (c >= C) return;
    const TA* cur_row = h + (size_t)t * C;
    const TA* old_row = t == first ? slot_row : cur_row - C;
    float cur[VEC], d[VEC];
    if (VEC == 8) {
        const uint4 a = *reinterpret_cast<const uint4*>(cur_row + c), b = *reinterpret_cast<const uint4*>(old_row + c);
        const TA* pa = reinterpret_cast<const TA*>(&a);
        const TA* pb = reinterpret_cast<const TA*>(&b);
#pragma unroll
        for (int i = 0; i < VEC; ++i) { cur[i] = to_f32(pa[i]); d[i] = to_f32(pb[i]) - cur[i]; }
        if (n == 1) *reinterpret_cast<uint4*>(slot_row + c) = a;
    } else {
        const TA a = cur_row[c];
        cur[0] = to_f32(a);
        d[0] = to_f32(old_row[c]) - cur[0];
        if (n == 1) slot_row[c] = a;
    }
    for (int s = 0; s < streams; ++s) {
        const float* m = mu + (size_t)s * C + c;
        TA* o = out + ((size_t)s * T + t) * C + c;
        if (VEC == 8) {
            const float4 m0 = *reinterpret_cast<const float4*>(m), m1 = *reinterpret_cast<const float4*>(m + 4);
            const float mm[8] = {m0.x, m0.y, m0.z, m0.w, m1.x, m1.y, m1.z, m1.w};
            uint4 r;
            TA* pr = reinterpret_cast<TA*>(&r);
#pragma unroll
            for (int i = 0; i < VEC; ++i) pr[i] = from_f32<TA>(fmaf(d[i], mm[i], cur[i]));
            *reinterpret_cast<uint4*>(o) = r;
        } else {
            o[0] = from_f32<TA>(fmaf(d[0], m[0], cur[0]));
        }
    }
}

// h [T, C] and state [slots, C] of one dtype; mu [streams, C] float; out [streams, T, C].
extern "C" int rb_token_shift(const void* h, void* state, const float* mu, void* out, int dtype, const int* cu_q, const int* tok_entry,
                              const int* entry_slot, int T, int C, int streams, void* stream) {
    if (T <= 0 || streams <= 0) return 0;
    if (C <= 0 || !cu_q || !tok_entry || !entry_slot) RB_REFUSE("token_shift: width %d, the entries' tables", C);
    cudaStream_t s = (cudaStream_t)stream;
    const bool vec = dtype == RB_BF16 && C % 8 == 0 && (((uintptr_t)h | (uintptr_t)state | (uintptr_t)mu | (uintptr_t)out) & 15) == 0;
    if (vec) return rb_launch(token_shift_kernel<bf16, 8>, dim3(T, rb_ceil_div(C, TS_THREADS * 8)), dim3(TS_THREADS), 0, s, (const bf16*)h, (bf16*)state, mu,
                              (bf16*)out, cu_q, tok_entry, entry_slot, T, C, streams);
    dim3 grid(T, rb_ceil_div(C, TS_THREADS));
    if (dtype == RB_BF16) return rb_launch(token_shift_kernel<bf16, 1>, grid, dim3(TS_THREADS), 0, s, (const bf16*)h, (bf16*)state, mu, (bf16*)out,
                                           cu_q, tok_entry, entry_slot, T, C, streams);
    if (dtype == RB_F32) return rb_launch(token_shift_kernel<float, 1>, grid, dim3(TS_THREADS), 0, s, (const float*)h, (float*)state, mu, (float*)out,
                                          cu_q, tok_entry, entry_slot, T, C, streams);
    RB_REFUSE("token_shift: dtype %d", dtype);
}

template <typename W>
__global__ void __launch_bounds__(TS_THREADS)
keep_last_rows_kernel(const W* __restrict__ rows, W* __restrict__ state, const int* __restrict__ cu_q, const int* __restrict__ entry_slot, int n) {
    pdl_trigger();
    const int e = blockIdx.y, i = blockIdx.x * TS_THREADS + threadIdx.x;
    const int end = cu_q[e + 1], len = end - cu_q[e];
    const int slot = entry_slot[e];
    pdl_wait();
    if (len > 1 && i < n) state[(size_t)slot * n + i] = rows[(size_t)(end - 1) * n + i];
}

extern "C" int rb_keep_last_rows(const void* rows, void* state, long long row_bytes, const int* cu_q, const int* entry_slot, int n_entries,
                                 void* stream) {
    if (n_entries <= 0 || row_bytes <= 0) return 0;
    if (n_entries > 65535 || row_bytes % 2 || row_bytes > (1LL << 30)) RB_REFUSE("keep_last_rows: %d entries, rows of %lld bytes", n_entries, row_bytes);
    cudaStream_t s = (cudaStream_t)stream;
    const uintptr_t at = (uintptr_t)rows | (uintptr_t)state | (uintptr_t)row_bytes;
#define KL_GO(W) do { const int n = (int)(row_bytes / (long long)sizeof(W)); \
        return rb_launch(keep_last_rows_kernel<W>, dim3(rb_ceil_div(n, TS_THREADS), n_entries), dim3(TS_THREADS), 0, s, (const W*)rows, (W*)state, cu_q, entry_slot, n); } while (0)
    if (at % 16 == 0) KL_GO(uint4);
    if (at % 4 == 0) KL_GO(uint32_t);
    KL_GO(uint16_t);
#undef KL_GO
}
