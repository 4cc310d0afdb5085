// Layer norm (or RMS norm) of rows, with what stands around it in one pass:
//
//   v = x[t] (+ alpha * delta[t]) (+ bias)          n = (v - mean) / sqrt(mean((v - mean)^2) + eps) * w     (RMS form: mean = 0)
//
// in front of a sublayer (`stream` null): out = n, and x takes v where delta is given and all rows are produced;
// behind a sublayer (`stream`): stream[t] += n, and out (if there is one) takes the stream's new row in the compute type.
// Statistics, sums and the stream are 32-bit; the mean is taken off before the squares are summed.
#include "common.cuh"

namespace {

// Sum over the CTA, the same for every thread, one barrier; `scratch` holds 32 floats and is used once.
__device__ __forceinline__ float row_sum(float v, float* scratch) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.f;
    for (int i = 0; i < (int)(blockDim.x + 31) >> 5; ++i) t += scratch[i];
    return t;
}

// four neighbouring elements a thread and turn, NV turns, the row in registers
template <int NV, bool CENTER, typename TO>
__global__ void __launch_bounds__(1024)
row_norm_kernel(float* __restrict__ x, const float* __restrict__ delta, float alpha, const float* __restrict__ bias, const float* __restrict__ w,
                float eps, const int* __restrict__ rows, float* __restrict__ stream, TO* __restrict__ out, int C) {
    __shared__ float scratch[2][32];
    pdl_trigger();
    pdl_wait();
    const int o = blockIdx.x, r = rows ? rows[o] : o;
    float v[NV][4];
    float sum = 0.f;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        const int i = (n * blockDim.x + threadIdx.x) * 4;
#pragma unroll
        for (int e = 0; e < 4; ++e) v[n][e] = 0.f;
        if (i < C) {
            load4(x + (size_t)r * C + i, v[n]);
            if (delta) {
                float d[4];
                load4(delta + (size_t)r * C + i, d);
#pragma unroll
                for (int e = 0; e < 4; ++e) v[n][e] = fmaf(alpha, d[e], v[n][e]);
            }
            if (bias) {
                float b[4];
                load4(bias + i, b);
#pragma unroll
                for (int e = 0; e < 4; ++e) v[n][e] += b[e];
            }
            if (delta && !rows && !stream) store4(x + (size_t)r * C + i, v[n]);
            sum += (v[n][0] + v[n][1]) + (v[n][2] + v[n][3]);
        }
    }
    const float mean = CENTER ? row_sum(sum, scratch[0]) / (float)C : 0.f;
    float ss = 0.f;
#pragma unroll
    for (int n = 0; n < NV; ++n)
        if ((int)(n * blockDim.x + threadIdx.x) * 4 < C)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                v[n][e] -= mean;
                ss = fmaf(v[n][e], v[n][e], ss);
            }
    const float scale = 1.f / sqrtf(row_sum(ss, scratch[1]) / (float)C + eps);
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        const int i = (n * blockDim.x + threadIdx.x) * 4;
        if (i >= C) continue;
        float wv[4];
        load4(w + i, wv);
#pragma unroll
        for (int e = 0; e < 4; ++e) v[n][e] = v[n][e] * scale * wv[e];
        if (stream) {
            float s[4];
            load4(stream + (size_t)r * C + i, s);
#pragma unroll
            for (int e = 0; e < 4; ++e) v[n][e] += s[e];
            store4(stream + (size_t)r * C + i, v[n]);
        }
        if (out) store4(out + (size_t)o * C + i, v[n]);
    }
}

// any size: the row waits in shared memory between the passes
template <bool CENTER, typename TO>
__global__ void __launch_bounds__(256)
row_norm_any_kernel(float* __restrict__ x, const float* __restrict__ delta, float alpha, const float* __restrict__ bias, const float* __restrict__ w,
                    float eps, const int* __restrict__ rows, float* __restrict__ stream, TO* __restrict__ out, int C) {
    extern __shared__ float row[];
    __shared__ float scratch[2][32];
    pdl_trigger();
    pdl_wait();
    const int o = blockIdx.x, r = rows ? rows[o] : o;
    float sum = 0.f;
    for (int i = threadIdx.x; i < C; i += blockDim.x) {
        float v = x[(size_t)r * C + i];
        if (delta) v = fmaf(alpha, delta[(size_t)r * C + i], v);
        if (bias) v += bias[i];
        if (delta && !rows && !stream) x[(size_t)r * C + i] = v;
        row[i] = v;
        sum += v;
    }
    const float mean = CENTER ? row_sum(sum, scratch[0]) / (float)C : 0.f;
    float ss = 0.f;
    for (int i = threadIdx.x; i < C; i += blockDim.x) {
        const float d = row[i] - mean;
        ss = fmaf(d, d, ss);
    }
    const float scale = 1.f / sqrtf(row_sum(ss, scratch[1]) / (float)C + eps);
    for (int i = threadIdx.x; i < C; i += blockDim.x) {
        float n = (row[i] - mean) * scale * w[i];
        if (stream) {
            n += stream[(size_t)r * C + i];
            stream[(size_t)r * C + i] = n;
        }
        if (out) out[(size_t)o * C + i] = from_float<TO>(n);
    }
}

template <bool CENTER, typename TO>
int go(float* x, const float* delta, float alpha, const float* bias, const float* w, float eps, const int* rows, float* stream, TO* out, int n, int C,
       cudaStream_t s) {
    const uintptr_t all = (uintptr_t)x | (uintptr_t)delta | (uintptr_t)bias | (uintptr_t)w | (uintptr_t)stream | (uintptr_t)out;
    if (C % 4 == 0 && all % 16 == 0 && C <= 4 * 1024 * 4) {
        const int quads = C / 4;
        // few rows: as many threads as quads, the shortest way through a row; many: four quads a thread, more rows on an SM
        const int nv = n <= 296 ? (quads <= 1024 ? 1 : quads <= 2048 ? 2 : 4) : (quads <= 64 ? 1 : quads <= 256 ? 2 : 4);
        const int threads = ((quads + nv - 1) / nv + 31) / 32 * 32;
        const dim3 grid(n), block(threads);
        if (nv == 1) return launch_pdl(row_norm_kernel<1, CENTER, TO>, grid, block, 0, s, x, delta, alpha, bias, w, eps, rows, stream, out, C);
        if (nv == 2) return launch_pdl(row_norm_kernel<2, CENTER, TO>, grid, block, 0, s, x, delta, alpha, bias, w, eps, rows, stream, out, C);
        return launch_pdl(row_norm_kernel<4, CENTER, TO>, grid, block, 0, s, x, delta, alpha, bias, w, eps, rows, stream, out, C);
    }
    const size_t smem = (size_t)C * sizeof(float);
    if (smem > 200 * 1024) return LLM_ERR_UNSUPPORTED;
    if (smem > 47 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(row_norm_any_kernel<CENTER, TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    return launch_pdl(row_norm_any_kernel<CENTER, TO>, dim3(n), dim3(256), smem, s, x, delta, alpha, bias, w, eps, rows, stream, out, C);
}

}  // namespace

// x [N, C], delta [N, C] (or null), bias [C] (or null), w [C], stream [N, C] (or null): float32.  rows (or null): the rows to be
// produced, out row o from row rows[o].  out: float32 or bfloat16, may be null with `stream`.  center: 1 layer norm, 0 RMS norm.
LLM_EXPORT int llm_row_norm(float* x, const float* delta, float alpha, const float* bias, const float* w, float eps, int center, const int* rows,
                            float* stream, void* out, int out_dtype, int n_out, int C, cudaStream_t s) {
    if (n_out <= 0) return 0;
    if (C <= 0 || !x || !w || (!out && !stream) || (stream && rows)) return LLM_ERR_BAD_ARGUMENT;
    if (out_dtype == LLM_F32)
        return center ? go<true, float>(x, delta, alpha, bias, w, eps, rows, stream, (float*)out, n_out, C, s)
                      : go<false, float>(x, delta, alpha, bias, w, eps, rows, stream, (float*)out, n_out, C, s);
    if (out_dtype == LLM_BF16)
        return center ? go<true, __nv_bfloat16>(x, delta, alpha, bias, w, eps, rows, stream, (__nv_bfloat16*)out, n_out, C, s)
                      : go<false, __nv_bfloat16>(x, delta, alpha, bias, w, eps, rows, stream, (__nv_bfloat16*)out, n_out, C, s);
    return LLM_ERR_BAD_ARGUMENT;
}
