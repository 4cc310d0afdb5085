// What a token's stacked projections become before softmax attention reads them as queries, keys and values.
//
// proj row: [Hq x D queries | Hk x D keys | Hk x V values]  (Hk = 0: a layer that reads another layer's keys and values;
// values_are_keys: no value columns, a key head's value is that head as projected, bias included, before norm and
// rotation).  In this order, each step optional:
//   bias:      the stacked bias (float32, laid out like the row) is added
//   norm:      1: every query head and every key head is divided by sqrt(mean(x^2) + eps) over its D lanes and multiplied
//              by qw / kw [D], the same for every head; 2: all query heads together are, over their Hq * D lanes, by
//              qw [Hq * D], all key heads likewise by kw [Hk * D]
//   rotate:    lanes i and i + rot/2 (i < rot/2) of every head turn by position * freq[i]; lanes >= rot pass
//              (interleaved: lanes 2i and 2i + 1 instead)
//   turn:      with v_freq [V / 2] every value head's pairs (lanes m and m + V/2, or 2m and 2m + 1) turn by
//              position * v_freq[m]; turn_out [N, V / 2] takes the (cos, sin) for whoever turns them back
//   values:    v_keep [N, Hk * V] (float32) takes the values as projected, bias included; or, with v_first [N, Hk * V],
//              the values become (1 - v_lambda) v + v_lambda v_first (those of the same token in an earlier layer)
//   warm:      queries times 1 + coef * ln(floor((position + 1) / every) + 1)
// Queries go to q_out [N, Hq * D]; keys and values into the token's slot of pool [pages, 2, Hk, page_size, Dp].  With maps = 2
// every two key heads in a row share a value head and a row of the pool [pages, 2, Hk / 2, page_size, Dp], side by side.
// Everything is computed in 32-bit.  One CTA per token, one warp per head at a time; where no head is normed by itself and
// everything lies on boundaries of four lanes, a second kernel takes four neighbouring pairs of lanes a thread instead.
#include <type_traits>

#include "common.cuh"

namespace {

constexpr int WARPS = 8;

template <typename TI, typename TQ, typename TK>
__global__ void __launch_bounds__(WARPS * 32)
head_prepare_kernel(const TI* __restrict__ proj, int ldp, const float* __restrict__ bias, TQ* __restrict__ q_out, int ldq,
                    TK* __restrict__ pool, const int* __restrict__ slot_map, int page_size, int Dp, const float* __restrict__ qw,
                    const float* __restrict__ kw, float eps, int normed, const float* __restrict__ freq, int rot,
                    const int* __restrict__ positions, float warm_coef, int warm_every, int Hq, int Hk, int D, int V,
                    int values_are_keys, int interleaved, float* __restrict__ v_keep, const float* __restrict__ v_first,
                    float v_lambda, int maps, const float* __restrict__ v_freq, float2* __restrict__ turn_out) {
    extern __shared__ float smem[];  // [WARPS][D] a head as projected, then rot/2 (cos, sin) pairs, then V/2 for the values
    __shared__ float scratch[33];
    float2* turn = reinterpret_cast<float2*>(smem + WARPS * D + ((WARPS * D) & 1));
    pdl_trigger();
    const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int half = rot >> 1;
    const int position = (half > 0 || warm_every > 0 || v_freq) ? positions[t] : 0;
    float2* v_turn = turn + half;
    const int v_half = v_freq ? V >> 1 : 0, Gv = Hk / maps;
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        float s, c;
        sincosf((float)position * freq[i], &s, &c);
        turn[i] = make_float2(c, s);
    }
    for (int i = threadIdx.x; i < v_half; i += blockDim.x) {
        float s, c;
        sincosf((float)position * v_freq[i], &s, &c);
        v_turn[i] = make_float2(c, s);
    }
    const float warm = warm_every > 0 ? 1.f + warm_coef * logf((float)((position + 1) / warm_every) + 1.f) : 1.f;
    const int slot = Hk > 0 ? slot_map[t] : 0;
    const int page = slot / page_size, off = slot % page_size;
    __syncthreads();
    pdl_wait();
    if (turn_out)
        for (int i = threadIdx.x; i < v_half; i += blockDim.x) turn_out[(size_t)t * v_half + i] = v_turn[i];
    const TI* row = proj + (size_t)t * ldp;
    float whole[2] = {1.f, 1.f};  // the scales of all query heads and of all key heads together
    if (normed == 2) {
        float sums[2] = {0.f, 0.f};
        for (int i = threadIdx.x; i < (Hq + Hk) * D; i += blockDim.x) {
            float v = to_float(row[i]);
            if (bias) v += bias[i];
            if (i < Hq * D) sums[0] = fmaf(v, v, sums[0]);
            else sums[1] = fmaf(v, v, sums[1]);
        }
        for (int e = 0; e < 2; ++e) {
            const float ss = block_sum(sums[e], scratch);
            whole[e] = 1.f / sqrtf(ss / (float)((e ? Hk : Hq) * D) + eps);
        }
    }
    float* buf = smem + warp * D;
    const int per_head = D - half;  // work items a head: `half` pairs, then the lanes that pass
    for (int head = warp; head < Hq + Hk; head += WARPS) {
        const bool is_q = head < Hq;
        const int base = head * D;  // keys follow the queries in the row and in the bias
        TK* vdst = (!is_q && values_are_keys) ? pool + ((((size_t)page * 2 + 1) * Hk + (head - Hq)) * page_size + off) * Dp : nullptr;  // (one map)
        float ss = 0.f;
        for (int d = lane; d < D; d += 32) {
            float v = to_float(row[base + d]);
            if (bias) v += bias[base + d];
            buf[d] = v;
            ss = fmaf(v, v, ss);
            if (vdst) vdst[d] = from_float<TK>(v);
        }
        ss = warp_sum(ss);
        const float ns = normed == 1 ? 1.f / sqrtf(ss / (float)D + eps) : normed == 2 ? whole[is_q ? 0 : 1] : 1.f;
        const float* w = normed ? (is_q ? qw : kw) : nullptr;
        if (normed == 2) w += (is_q ? head : head - Hq) * D;
        const float post = is_q ? warm : 1.f;
        __syncwarp();
        for (int i = lane; i < per_head; i += 32) {
            float a, b = 0.f;
            int da, db = -1;
            if (i < half) {
                da = interleaved ? 2 * i : i; db = interleaved ? 2 * i + 1 : i + half;
                float u = buf[da] * ns, v = buf[db] * ns;
                if (w) { u *= w[da]; v *= w[db]; }
                const float c = turn[i].x, s = turn[i].y;
                a = (u * c - v * s) * post;
                b = (v * c + u * s) * post;
            } else {
                da = i + half;
                float u = buf[da] * ns;
                if (w) u *= w[da];
                a = u * post;
            }
            if (is_q) {
                TQ* dst = q_out + (size_t)t * ldq + base;
                dst[da] = from_float<TQ>(a);
                if (db >= 0) dst[db] = from_float<TQ>(b);
            } else {
                const int kh = (head - Hq) / maps;
                TK* dst = pool + (((size_t)page * 2 * Gv + kh) * page_size + off) * Dp + (head - Hq - kh * maps) * D;
                dst[da] = from_float<TK>(a);
                if (db >= 0) dst[db] = from_float<TK>(b);
            }
        }
        __syncwarp();
    }
    if (Hk > 0 && !values_are_keys) {
        const int vbase = (Hq + Hk) * D;
        if (v_freq) {
            for (int i = threadIdx.x; i < Gv * v_half; i += blockDim.x) {
                const int kh = i / v_half, m = i - kh * v_half;
                const int da = interleaved ? 2 * m : m, db = interleaved ? 2 * m + 1 : m + v_half;
                float u = to_float(row[vbase + kh * V + da]), v = to_float(row[vbase + kh * V + db]);
                if (bias) { u += bias[vbase + kh * V + da]; v += bias[vbase + kh * V + db]; }
                const float2 cs = v_turn[m];
                TK* dst = pool + ((((size_t)page * 2 + 1) * Gv + kh) * page_size + off) * Dp;
                dst[da] = from_float<TK>(u * cs.x - v * cs.y);
                dst[db] = from_float<TK>(v * cs.x + u * cs.y);
            }
            return;
        }
        for (int i = threadIdx.x; i < Gv * V; i += blockDim.x) {
            const int kh = i / V, d = i % V;
            float v = to_float(row[vbase + i]);
            if (bias) v += bias[vbase + i];
            if (v_keep) v_keep[(size_t)t * Gv * V + i] = v;
            if (v_first) v = (1.f - v_lambda) * v + v_lambda * v_first[(size_t)t * Gv * V + i];
            pool[((((size_t)page * 2 + 1) * Gv + kh) * page_size + off) * Dp + d] = from_float<TK>(v);
        }
    }
}

// No norm, or one over whole projections; half layout; no factor on the queries, no values kept or mixed; D, rot / 2, V (and V / 2
// where the values turn), the pitches and Dp multiples of four.  A thread takes four neighbouring pairs of a head, or four lanes
// that pass, at a time (16-byte loads, 8- or 16-byte stores).  Grid (tokens, shares): a token's items may be shared out over several
// CTAs (steps of few tokens), each of which works out the token's angles and sums for itself.
template <typename TO>
__global__ void __launch_bounds__(256)
head_prepare_wide_kernel(const float* __restrict__ proj, int ldp, const float* __restrict__ bias, TO* __restrict__ q_out, int ldq,
                         TO* __restrict__ pool, const int* __restrict__ slot_map, int page_size, int Dp, const float* __restrict__ qw,
                         const float* __restrict__ kw, float eps, const float* __restrict__ freq, int rot, const int* __restrict__ positions,
                         int Hq, int Hk, int D, int V, int maps, const float* __restrict__ v_freq, float2* __restrict__ turn_out) {
    extern __shared__ float2 turn[];  // rot / 2 (cos, sin), then V / 2 for the values
    __shared__ float scratch[33];
    pdl_trigger();
    const int t = blockIdx.x, half = rot >> 1, v_half = v_freq ? V >> 1 : 0, Gv = Hk / maps;
    const float position = half + v_half > 0 ? (float)positions[t] : 0.f;
    for (int i = threadIdx.x; i < half + v_half; i += blockDim.x) {
        float s, c;
        sincosf(position * (i < half ? freq[i] : v_freq[i - half]), &s, &c);
        turn[i] = make_float2(c, s);
    }
    const int slot = Hk > 0 ? slot_map[t] : 0;
    const int page = slot / page_size, off = slot - page * page_size;
    __syncthreads();
    pdl_wait();
    if (turn_out && blockIdx.y == 0)
        for (int i = threadIdx.x; i < v_half; i += blockDim.x) turn_out[(size_t)t * v_half + i] = turn[half + i];
    const float* row = proj + (size_t)t * ldp;
    auto load = [&](int c, float (&v)[4]) {
        load4(row + c, v);
        if (bias) {
            float b[4];
            load4(bias + c, b);
#pragma unroll
            for (int e = 0; e < 4; ++e) v[e] += b[e];
        }
    };
    float whole[2] = {1.f, 1.f};
    if (qw) {
        float sums[2] = {0.f, 0.f};
        for (int c = threadIdx.x * 4; c < (Hq + Hk) * D; c += blockDim.x * 4) {
            float v[4];
            load(c, v);
            const float s = fmaf(v[0], v[0], v[1] * v[1]) + fmaf(v[2], v[2], v[3] * v[3]);
            if (c < Hq * D) sums[0] += s;
            else sums[1] += s;
        }
#pragma unroll
        for (int e = 0; e < 2; ++e) whole[e] = 1.f / sqrtf(block_sum(sums[e], scratch) / (float)((e ? Hk : Hq) * D) + eps);
    }
    const int pairs = half >> 2, per = pairs + ((D - rot) >> 2), per_v = v_half > 0 ? v_half >> 2 : V >> 2;
    const int heads_items = (Hq + Hk) * per, items = heads_items + Gv * per_v;
    for (int it = blockIdx.y * blockDim.x + threadIdx.x; it < items; it += gridDim.y * blockDim.x) {
        const bool is_v = it >= heads_items;
        const int local = is_v ? it - heads_items : it, span = is_v ? per_v : per;
        const int head = local / span, i = local - head * span;
        const bool turns = is_v ? v_half > 0 : i < pairs;
        const int da = turns ? 4 * i : is_v ? 4 * i : 4 * i + half;  // (lanes that pass follow the rotated ones: rot + 4 (i - pairs))
        const int src = is_v ? (Hq + Hk) * D + head * V : head * D;
        float a[4], b[4];
        load(src + da, a);
        if (turns) load(src + da + (is_v ? v_half : half), b);
        if (!is_v && qw) {
            const bool is_q = head < Hq;
            const float* w = is_q ? qw + head * D : kw + (head - Hq) * D;
            const float s = whole[is_q ? 0 : 1];
            float x[4];
            load4(w + da, x);
#pragma unroll
            for (int e = 0; e < 4; ++e) a[e] = a[e] * s * x[e];
            if (turns) {
                load4(w + da + half, x);
#pragma unroll
                for (int e = 0; e < 4; ++e) b[e] = b[e] * s * x[e];
            }
        }
        TO* dst;
        if (is_v) dst = pool + ((((size_t)page * 2 + 1) * Gv + head) * page_size + off) * Dp;
        else if (head < Hq) dst = q_out + (size_t)t * ldq + head * D;
        else {
            const int k = head - Hq, kh = k / maps;
            dst = pool + (((size_t)page * 2 * Gv + kh) * page_size + off) * Dp + (k - kh * maps) * D;
        }
        if (turns) {
            const float2* cs = turn + (is_v ? half : 0) + 4 * i;
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float u = a[e], v = b[e];
                a[e] = u * cs[e].x - v * cs[e].y;
                b[e] = v * cs[e].x + u * cs[e].y;
            }
            store4(dst + da + (is_v ? v_half : half), b);
        }
        store4(dst + da, a);
    }
}

}  // namespace

// in_dtype: the projections' type; out_dtype: the type of the queries on their way out and of the pool.
LLM_EXPORT int llm_head_prepare(const void* proj, int in_dtype, int ldp, const float* bias, void* q_out, int ldq, void* pool,
                                int out_dtype, const int* slot_map, int page_size, int Dp, const float* qw, const float* kw, float eps,
                                int normed, const float* freq, int rot, const int* positions, float warm_coef, int warm_every, int N,
                                int Hq, int Hk, int D, int V, int values_are_keys, int interleaved, float* v_keep,
                                const float* v_first, float v_lambda, int maps, const float* v_freq, void* turn_out, cudaStream_t stream) {
    if (N <= 0) return 0;
    if (maps < 1 || Hk % maps || (maps > 1 && values_are_keys) || normed < 0 || normed > 2 ||
        (v_freq && (V & 1 || values_are_keys || Hk <= 0 || v_keep || v_first || !positions)) || (turn_out && !v_freq))
        return LLM_ERR_BAD_ARGUMENT;
    if (rot < 0 || rot % 2 || rot > D || Hq < 0 || Hk < 0 || D <= 0 || D > 1024 || (Hk > 0 && (!pool || !slot_map || Dp < maps * D || page_size <= 0)) ||
        (Hk > 0 && !values_are_keys && (V <= 0 || Dp < V)) || ((rot > 0 || warm_every > 0) && !positions) || (rot > 0 && !freq) ||
        (normed && (!qw || (Hk > 0 && !kw))) || (Hq > 0 && !q_out) || ((v_keep || v_first) && (values_are_keys || Hk <= 0)))
        return LLM_ERR_BAD_ARGUMENT;
    using bf = __nv_bfloat16;
    auto aligned = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
    const int v_lanes = v_freq ? V / 2 : V;
    if (in_dtype == LLM_F32 && normed != 1 && !interleaved && !values_are_keys && warm_every <= 0 && !v_keep && !v_first &&
        ((D | (rot / 2) | (Hk > 0 ? v_lanes | Dp : 0) | ldp | ldq) & 3) == 0 && aligned(proj) && aligned(bias) && aligned(q_out) && aligned(pool) &&
        aligned(qw) && aligned(kw)) {
        const int items = (Hq + Hk) * (D / 4 - rot / 8) + (Hk / maps) * (v_lanes / 4);
        int shares = (2 * 148 + N - 1) / N, most = (items + 255) / 256;
        if (shares > most) shares = most;
        const size_t wide_smem = (size_t)(rot / 2 + (v_freq ? V / 2 : 0) + 1) * sizeof(float2);
        auto wide = [&](auto kernel, auto* qo) {
            using TO = std::remove_pointer_t<decltype(qo)>;
            return launch_pdl(kernel, dim3(N, shares < 1 ? 1 : shares), dim3(256), wide_smem, stream, (const float*)proj, ldp, bias, qo, ldq, (TO*)pool,
                              slot_map, page_size, Dp, normed ? qw : nullptr, kw, eps, freq, rot, positions, Hq, Hk, D, V, maps, v_freq, (float2*)turn_out);
        };
        if (out_dtype == LLM_F32) return wide(head_prepare_wide_kernel<float>, (float*)q_out);
        if (out_dtype == LLM_BF16) return wide(head_prepare_wide_kernel<bf>, (bf*)q_out);
    }
    const size_t smem = ((size_t)WARPS * D + 1) * sizeof(float) + (size_t)(rot / 2 + 1 + (v_freq ? V / 2 : 0)) * sizeof(float2);
    auto go = [&](auto kernel, auto* in, auto* qo) {
        using TK = std::remove_pointer_t<decltype(qo)>;
        return launch_pdl(kernel, dim3(N), dim3(WARPS * 32), smem, stream, in, ldp, bias, qo, ldq, (TK*)pool, slot_map, page_size, Dp, qw, kw,
                          eps, normed, freq, rot, positions, warm_coef, warm_every, Hq, Hk, D, V, values_are_keys, interleaved, v_keep, v_first, v_lambda, maps, v_freq,
                          (float2*)turn_out);
    };
    if (in_dtype == LLM_F32 && out_dtype == LLM_F32) return go(head_prepare_kernel<float, float, float>, (const float*)proj, (float*)q_out);
    if (in_dtype == LLM_F32 && out_dtype == LLM_BF16) return go(head_prepare_kernel<float, bf, bf>, (const float*)proj, (bf*)q_out);
    if (in_dtype == LLM_BF16 && out_dtype == LLM_BF16) return go(head_prepare_kernel<bf, bf, bf>, (const bf*)proj, (bf*)q_out);
    return LLM_ERR_UNSUPPORTED;
}
