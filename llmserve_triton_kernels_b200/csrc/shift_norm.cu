// Two RMS norms of one residual stream, for layers whose mixer and feed-forward read the same rows side by side, with a token
// shift on the first.
//
//   n_t = x_t / sqrt(mean(x_t^2) + eps)
//   out1_t = h_t + shift * (h_(t-1) - h_t),  h_t = n_t * w1      (shift null: out1_t = h_t)
//   out2_t = n_t * w2                                            (w2 null: not written)
//
// h_(t-1) is the row of the token in front in the same request: a row of this step, or for a request's first token of the step the
// request's slot of `state` [slots, W] (float32: h of the last token that earlier steps brought, zeros at a request's start).
// The CTA that handles a request's first token of the step reads the slot and then moves it on to h of the request's last token
// of the step, which it computes once more: no other CTA touches the slot, so nothing has to wait.  Statistics, norms, the
// shift and the state are 32-bit, and a row's sum of squares has an order that depends on W alone.
#include "common.cuh"

namespace {

struct ShiftNormArgs {
    const float* x;  // [N, W]
    const float *w1, *w2, *shift;
    float eps;
    float* state;
    const int *state_slots, *token_request, *cu_tokens;
    int N, W, span;
};

// A CTA walks `span` tokens with its part of a row in registers (NV pieces of four lanes a thread), h of the token in front kept
// from token to token and the next row asked for while the present one is summed.
template <typename TO, int NV>
__global__ void __launch_bounds__(256) shift_norm_kernel(const ShiftNormArgs a, TO* __restrict__ out1, TO* __restrict__ out2) {
    __shared__ float scratch[33];
    pdl_trigger();
    const int W = a.W, c0 = threadIdx.x * 4, step = blockDim.x * 4;
    float w1[NV][4], w2[NV][4], sh[NV][4];
#pragma unroll
    for (int j = 0; j < NV; ++j) {
        const int c = c0 + j * step;
        if (c < W) {
            load4(a.w1 + c, w1[j]);
            if (out2) load4(a.w2 + c, w2[j]);
            if (a.shift) load4(a.shift + c, sh[j]);
        }
    }
    const int t0 = blockIdx.x * a.span, t1 = min(a.N, t0 + a.span);
    int r = 0, begin = 0, end = 0;
    if (a.shift) {
        r = a.token_request[t0];
        begin = a.cu_tokens[r];
        end = a.cu_tokens[r + 1];
    }
    pdl_wait();
    auto fetch = [&](int t, float (&v)[NV][4]) {
#pragma unroll
        for (int j = 0; j < NV; ++j)
            if (c0 + j * step < W) load4(a.x + (size_t)t * W + c0 + j * step, v[j]);
    };
    auto scale_of = [&](const float (&v)[NV][4]) {
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < NV; ++j)
            if (c0 + j * step < W) {
#pragma unroll
                for (int e = 0; e < 4; ++e) ss = fmaf(v[j][e], v[j][e], ss);
            }
        return 1.f / sqrtf(block_sum(ss, scratch) / (float)W + a.eps);
    };
    float next[NV][4], before[NV][4];
    if (a.shift && t0 > begin) {  // h of the row in front of the first
        fetch(t0 - 1, before);
        fetch(t0, next);
        const float s = scale_of(before);
#pragma unroll
        for (int j = 0; j < NV; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) before[j][e] = before[j][e] * s * w1[j][e];
    } else {
        fetch(t0, next);
    }
    for (int t = t0; t < t1; ++t) {
        if (a.shift && t == end) {
            ++r;
            begin = end;
            end = a.cu_tokens[r + 1];
        }
        float v[NV][4];
#pragma unroll
        for (int j = 0; j < NV; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) v[j][e] = next[j][e];
        const bool first = a.shift && t == begin;
        float* slot = first ? a.state + (size_t)a.state_slots[r] * W : nullptr;
        if (first) {
#pragma unroll
            for (int j = 0; j < NV; ++j)
                if (c0 + j * step < W) load4(slot + c0 + j * step, before[j]);
        }
        if (t + 1 < t1) fetch(t + 1, next);
        const float s = scale_of(v);
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int c = c0 + j * step;
            if (c < W) {
                float y[4];
                if (out2) {
#pragma unroll
                    for (int e = 0; e < 4; ++e) y[e] = v[j][e] * s * w2[j][e];
                    store4(out2 + (size_t)t * W + c, y);
                }
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float h = v[j][e] * s * w1[j][e];
                    y[e] = a.shift ? fmaf(sh[j][e], before[j][e] - h, h) : h;
                    before[j][e] = h;
                }
                store4(out1 + (size_t)t * W + c, y);
            }
        }
        if (first) {  // the slot moves on to h of the request's last token of this step
            float last[NV][4];
            float ls = 1.f;
            if (end - 1 > t) {
                fetch(end - 1, last);
                ls = scale_of(last);
            }
#pragma unroll
            for (int j = 0; j < NV; ++j) {
                const int c = c0 + j * step;
                if (c < W) {
                    float y[4];
#pragma unroll
                    for (int e = 0; e < 4; ++e) y[e] = end - 1 > t ? last[j][e] * ls * w1[j][e] : before[j][e];
                    store4(slot + c, y);
                }
            }
        }
    }
}

// Any row length and any alignment: a CTA a token, rows read twice.
template <typename TO>
__global__ void __launch_bounds__(256) shift_norm_any_kernel(const ShiftNormArgs a, TO* __restrict__ out1, TO* __restrict__ out2) {
    __shared__ float scratch[33];
    pdl_trigger();
    const int t = blockIdx.x, W = a.W;
    int r = 0, begin = 0, end = 0;
    if (a.shift) {
        r = a.token_request[t];
        begin = a.cu_tokens[r];
        end = a.cu_tokens[r + 1];
    }
    pdl_wait();
    auto scale_of = [&](int row) {
        const float* x = a.x + (size_t)row * W;
        float ss = 0.f;
        for (int i = threadIdx.x; i < W; i += blockDim.x) ss = fmaf(x[i], x[i], ss);
        return 1.f / sqrtf(block_sum(ss, scratch) / (float)W + a.eps);
    };
    const float* x = a.x + (size_t)t * W;
    const float s = scale_of(t);
    const bool first = a.shift && t == begin, from_row = a.shift && t > begin;
    float* slot = first ? a.state + (size_t)a.state_slots[r] * W : nullptr;
    const float ps = from_row ? scale_of(t - 1) : 1.f;
    const bool more = first && end - 1 > t;
    const float ls = more ? scale_of(end - 1) : 1.f;
    for (int i = threadIdx.x; i < W; i += blockDim.x) {
        const float w = a.w1[i], h = x[i] * s * w;
        float y = h;
        if (a.shift) {
            const float before = first ? slot[i] : x[i - W] * ps * w;
            y = fmaf(a.shift[i], before - h, h);
        }
        out1[(size_t)t * W + i] = from_float<TO>(y);
        if (out2) out2[(size_t)t * W + i] = from_float<TO>(x[i] * s * a.w2[i]);
        if (first) slot[i] = more ? a.x[(size_t)(end - 1) * W + i] * ls * w : h;
    }
}

template <typename TO>
int shift_norm_launch(ShiftNormArgs a, TO* out1, TO* out2, cudaStream_t stream) {
    auto aligned = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
    const bool wide = (a.W & 3) == 0 && a.W <= 8192 && aligned(a.x) && aligned(a.w1) && aligned(a.w2) && aligned(a.shift) && aligned(a.state) &&
                      aligned(out1) && aligned(out2);
    if (!wide) return launch_pdl(shift_norm_any_kernel<TO>, dim3(a.N), dim3(256), 0, stream, a, out1, out2);
    const int quads = a.W / 4, threads = quads >= 256 ? 256 : (quads + 31) / 32 * 32;
    // long steps: a few tokens a CTA (the row in front of a CTA's first is read once more), as long as every SM has several CTAs
    const int most = a.N / (148 * 4);
    a.span = most < 1 ? 1 : most > 16 ? 16 : most;
    const dim3 grid((a.N + a.span - 1) / a.span);
    const int pieces = (quads + threads - 1) / threads;
    if (pieces <= 1) return launch_pdl(shift_norm_kernel<TO, 1>, grid, dim3(threads), 0, stream, a, out1, out2);
    if (pieces <= 2) return launch_pdl(shift_norm_kernel<TO, 2>, grid, dim3(threads), 0, stream, a, out1, out2);
    if (pieces <= 4) return launch_pdl(shift_norm_kernel<TO, 4>, grid, dim3(threads), 0, stream, a, out1, out2);
    return launch_pdl(shift_norm_kernel<TO, 8>, grid, dim3(threads), 0, stream, a, out1, out2);
}

}  // namespace

// x [N, W] float32 contiguous -> out1, out2 [N, W] of type out_dtype (out2 null: one norm).  shift [W] null: no token shift (state,
// state_slots, token_request and cu_tokens are then not read).
LLM_EXPORT int llm_shift_norm(const float* x, const float* w1, const float* w2, const float* shift, float eps, float* state,
                              const int* state_slots, const int* token_request, const int* cu_tokens, void* out1, void* out2,
                              int out_dtype, int N, int W, cudaStream_t stream) {
    if (N <= 0) return 0;
    if (W <= 0 || !x || !w1 || !out1 || (out2 && !w2) || (shift && (!state || !state_slots || !token_request || !cu_tokens))) return LLM_ERR_BAD_ARGUMENT;
    ShiftNormArgs a = {x, w1, w2, shift, eps, state, state_slots, token_request, cu_tokens, N, W, 1};
    if (out_dtype == LLM_F32) return shift_norm_launch<float>(a, (float*)out1, (float*)out2, stream);
    if (out_dtype == LLM_BF16) return shift_norm_launch<__nv_bfloat16>(a, (__nv_bfloat16*)out1, (__nv_bfloat16*)out2, stream);
    return LLM_ERR_BAD_ARGUMENT;
}
