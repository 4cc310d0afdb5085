// The gated delta rule: a matrix of state per (request, head) that forgets by a factor of the token's choosing and is
// corrected towards the token's value at the token's key.
//
//   S <- g_t S        u_t = beta_t (v_t - S^T k_t)        S <- S + k_t u_t^T        o_t = S^T q_t         S: [D, V] float32
//   k_t, q_t: unit vectors x / sqrt(sum x^2 + 1e-6), q_t times q_scale       beta_t = sigmoid(b_t)
//   g_t = exp(-exp(A_log_h) * softplus(a_t + dt_bias_h))
//
// Everything is 32-bit.  q and k have G heads, v, beta and g have H; head h reads q/k head h / (H / G).  Column v of S is all
// that u_t[v] and o_t[v] need, so columns are shared out.  Two ways:
//
// Few tokens a request (decode steps): delta_step_kernel, one CTA a (request, head) with the whole state in registers, which
// also norms the head's o, weighs and gates it.  With r = S_old^T q the read-out is o = g r + (k . q) u, so that both sums
// over the old state are taken in one pass.
//
// Prompts: eight tokens at a time.  With L_t the sum of ln g over the block's tokens up to t, G_t = exp(L_t) and S the state
// in front of the block,
//
//   u_t = beta_t (v_t - G_t S^T k_t - sum_(i<t) exp(L_t - L_i) (k_t . k_i) u_i)
//   o_t = G_t S^T q_t + sum_(i<=t) exp(L_t - L_i) (q_t . k_i) u_i
//   S_after = G_7 S + sum_i exp(L_7 - L_i) k_i u_i^T
//
// The first line is a triangular system (I + A) u = beta (v - G S^T k) whose matrix does not know the state: M = (I + A)^-1 diag(beta).
// delta_prepare_kernel makes the unit vectors, M, P (the second line's factors), G and E_i = exp(L_7 - L_i) for every block of
// every request, all blocks at once; delta_scan_kernel walks the blocks: the dots with S, u = M (v - G dots), o, and the update.
#include "common.cuh"

namespace {

constexpr int BLK = 8;     // tokens a block
constexpr int COEF = 144;  // floats a (block, head): M [8][8], P [8][8], G [8], E [8]
constexpr int GROUPS = 16; // groups of threads a CTA of the scan: each owns some neighbouring columns of the state
constexpr int TPC = 8;     // threads a group: each holds D / 8 rows of the group's columns

__device__ __forceinline__ void copy16(float* smem, const float* gmem) {
    const unsigned dst = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(dst), "l"(gmem));
}

__device__ __forceinline__ float log_decay(float a, float dt_bias, float a_log) {
    const float z = a + dt_bias;
    return -expf(a_log) * (fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))));
}

__device__ __forceinline__ float sigmoid_of(float z) { return 1.f / (1.f + expf(-z)); }

// The index of a request's first block among all blocks of the step: blocks of different requests never share one.
__device__ __forceinline__ int first_block(int begin, int r) { return begin / BLK + r; }

// grid (blocks of the longest request, G, requests), 128 threads.  y: rows [q: G*D | k: G*D | ...] (pitch ldy), q and k made
// unit vectors in place.  coef: [blocks, H, COEF]
__global__ void __launch_bounds__(128)
delta_prepare_kernel(float* __restrict__ y, int ldy, const float* __restrict__ b, int ldb, const float* __restrict__ a, int lda,
                     const float* __restrict__ a_log, const float* __restrict__ dt_bias, const int* __restrict__ cu_tokens,
                     float* __restrict__ coef, int G, int H, int D, float q_scale) {
    extern __shared__ __align__(16) float shared[];
    __shared__ float dots[2][BLK][BLK];  // k_t . k_i and q_t . k_i
    pdl_trigger();
    const int r = blockIdx.z, g = blockIdx.y, rep = H / G;
    const int request = cu_tokens[r], end = cu_tokens[r + 1], begin = request + blockIdx.x * BLK;
    if (begin >= end) return;
    const int count = min(BLK, end - begin);
    const int D4 = (D + 3) & ~3, pitch = D4 + 4;
    float* sk = shared;              // [8][pitch]
    float* sq = shared + BLK * pitch;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    pdl_wait();
    for (int t = warp * 2; t < warp * 2 + 2; ++t) {
        float* qrow = y + (size_t)(begin + t) * ldy + (size_t)g * D;
        float* krow = qrow + (size_t)G * D;
        float qq = 0.f, kk = 0.f;
        for (int d = lane; d < D4; d += 32) {
            const float qv = t < count && d < D ? qrow[d] : 0.f, kv = t < count && d < D ? krow[d] : 0.f;
            sq[t * pitch + d] = qv;
            sk[t * pitch + d] = kv;
            qq = fmaf(qv, qv, qq);
            kk = fmaf(kv, kv, kk);
        }
        const float fq = q_scale / sqrtf(warp_sum(qq) + 1e-6f), fk = 1.f / sqrtf(warp_sum(kk) + 1e-6f);
        for (int d = lane; d < D; d += 32) {
            const float qv = sq[t * pitch + d] * fq, kv = sk[t * pitch + d] * fk;
            sq[t * pitch + d] = qv;
            sk[t * pitch + d] = kv;
            if (t < count) {
                qrow[d] = qv;
                krow[d] = kv;
            }
        }
    }
    __syncthreads();
    {
        const int which = threadIdx.x >> 6, t = (threadIdx.x >> 3) & 7, i = threadIdx.x & 7;
        if (i <= t) {
            const float* x = (which ? sq : sk) + t * pitch;
            const float* z = sk + i * pitch;
            float s0 = 0.f, s1 = 0.f;
            for (int d = 0; d < D4; d += 4) {
                const float4 xv = *reinterpret_cast<const float4*>(x + d), zv = *reinterpret_cast<const float4*>(z + d);
                s0 = fmaf(xv.x, zv.x, s0);
                s1 = fmaf(xv.y, zv.y, s1);
                s0 = fmaf(xv.z, zv.z, s0);
                s1 = fmaf(xv.w, zv.w, s1);
            }
            dots[which][t][i] = s0 + s1;
        } else dots[which][t][i] = 0.f;
    }
    __syncthreads();
    const int j = threadIdx.x & 7;
    const unsigned mask = 0xffu << (threadIdx.x & 24);
    for (int hh = threadIdx.x >> 3; hh < rep; hh += 16) {  // eight threads a head: thread j has token j, column j of M, row j of P
        const int h = g * rep + hh;
        float L = 0.f, beta = 0.f;
        if (j < count) {
            L = log_decay(a[(size_t)(begin + j) * lda + h], dt_bias[h], a_log[h]);
            beta = sigmoid_of(b[(size_t)(begin + j) * ldb + h]);
        }
#pragma unroll
        for (int o = 1; o < 8; o <<= 1) {
            const float up = __shfl_up_sync(mask, L, o, 8);
            if (j >= o) L += up;
        }
        float Ls[BLK], betas[BLK];
#pragma unroll
        for (int t = 0; t < BLK; ++t) {
            Ls[t] = __shfl_sync(mask, L, t, 8);
            betas[t] = __shfl_sync(mask, beta, t, 8);
        }
        float* to = coef + ((size_t)(first_block(request, r) + blockIdx.x) * H + h) * COEF;
        float T[BLK];  // column j of (I + A)^-1
#pragma unroll
        for (int t = 0; t < BLK; ++t) {
            float s = 0.f;
#pragma unroll
            for (int i = 0; i < t; ++i) s = fmaf(betas[t] * expf(Ls[t] - Ls[i]) * dots[0][t][i], T[i], s);
            T[t] = t < j ? 0.f : t == j ? 1.f : -s;
            to[t * BLK + j] = T[t] * beta;
        }
        for (int i = 0; i < BLK; ++i) to[64 + j * BLK + i] = i <= j ? expf(L - Ls[i]) * dots[1][j][i] : 0.f;
        to[128 + j] = expf(L);
        to[136 + j] = j < count ? expf(Ls[BLK - 1] - L) : 0.f;
    }
}

// Eight lanes hold partial sums of eight tokens; they trade halves (4, 2, 1 values) so that lane `sub` ends with token sub's sum.
__device__ __forceinline__ float trade_sum(const float (&o)[BLK], int sub) {
    const bool h4 = sub & 4, h2 = sub & 2, h1 = sub & 1;
    float a[4], b[2];
#pragma unroll
    for (int u = 0; u < 4; ++u) a[u] = (h4 ? o[u + 4] : o[u]) + __shfl_xor_sync(0xffffffffu, h4 ? o[u] : o[u + 4], 4);
#pragma unroll
    for (int u = 0; u < 2; ++u) b[u] = (h2 ? a[u + 2] : a[u]) + __shfl_xor_sync(0xffffffffu, h2 ? a[u] : a[u + 2], 2);
    return (h1 ? b[1] : b[0]) + __shfl_xor_sync(0xffffffffu, h1 ? b[0] : b[1], 1);
}

// grid (columns of V, H, requests), 128 threads: 16 groups of 8, CPT neighbouring columns a group, DPT rows a thread.
// q, k, v: columns of y's rows (unit vectors made by the kernel above); coef as above; out: [N, H, V] float32
template <int DPT, int TB, int CPT>
__global__ void __launch_bounds__(GROUPS * TPC)
delta_scan_kernel(const float* __restrict__ q, const float* __restrict__ k, const float* __restrict__ v, int ld, const float* __restrict__ coef,
                  float* __restrict__ states, const int* __restrict__ state_slots, const int* __restrict__ cu_tokens, float* __restrict__ out,
                  int H, int G, int D, int V) {
    constexpr int COLS = GROUPS * CPT;
    constexpr int DS = DPT * TPC;   // rows that the CTA's registers have room for (>= D)
    constexpr int SEG = DPT + 4;    // a part's lanes of a token's q or k, then 4 floats of room: the parts' 16-byte reads fall
    constexpr int RP = SEG * TPC;   // into different banks; RP: the pitch of a token's row
    constexpr int NB = TB / BLK;
    extern __shared__ __align__(16) float shared[];
    float* sq = shared;                   // [2][TB][RP]
    float* sk = sq + 2 * TB * RP;         // [2][TB][RP]
    float* sv = sk + 2 * TB * RP;         // [2][TB][COLS]
    float* sc = sv + 2 * TB * COLS;       // [2][NB][COEF]
    float* tile = sc + 2 * NB * COEF;     // [DS][COLS + 1], the state on its way in and out
    pdl_trigger();
    const int r = blockIdx.z, h = blockIdx.y, v0 = blockIdx.x * COLS, g = h / (H / G);
    const int sub = threadIdx.x % TPC, c0 = (threadIdx.x / TPC) * CPT;
    const int begin = cu_tokens[r], end = cu_tokens[r + 1], slot = state_slots[r], block0 = first_block(begin, r);
    float* state = states + ((size_t)slot * H + h) * D * V;
    const bool vec = D % 4 == 0 && ld % 4 == 0 && (reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k)) % 16 == 0;
    const bool vec_v = V % 4 == 0 && ld % 4 == 0 && reinterpret_cast<uintptr_t>(v) % 16 == 0 && v0 + COLS <= V;
    pdl_wait();
    if (begin >= end) return;

    auto fetch = [&](int t0, int buf) {
        const int count = min(TB, end - t0), whole = (count + BLK - 1) / BLK * BLK;
        if (vec) {
            const int chunks = D / 4;
            for (int i = threadIdx.x; i < count * chunks; i += blockDim.x) {
                const int tt = i / chunks, d = (i % chunks) * 4;
                const size_t at = ((size_t)buf * TB + tt) * RP + (d / DPT) * SEG + d % DPT;
                copy16(sq + at, q + (size_t)(t0 + tt) * ld + (size_t)g * D + d);
                copy16(sk + at, k + (size_t)(t0 + tt) * ld + (size_t)g * D + d);
            }
        } else {
            for (int i = threadIdx.x; i < count * D; i += blockDim.x) {
                const int tt = i / D, d = i % D;
                const size_t at = ((size_t)buf * TB + tt) * RP + (d / DPT) * SEG + d % DPT;
                sq[at] = q[(size_t)(t0 + tt) * ld + (size_t)g * D + d];
                sk[at] = k[(size_t)(t0 + tt) * ld + (size_t)g * D + d];
            }
        }
        if (vec_v) {
            for (int i = threadIdx.x; i < count * (COLS / 4); i += blockDim.x) {
                const int tt = i / (COLS / 4), c = (i % (COLS / 4)) * 4;
                copy16(sv + ((size_t)buf * TB + tt) * COLS + c, v + (size_t)(t0 + tt) * ld + (size_t)h * V + v0 + c);
            }
        } else {
            for (int i = threadIdx.x; i < count * COLS; i += blockDim.x) {
                const int tt = i / COLS, c = i % COLS;
                sv[((size_t)buf * TB + tt) * COLS + c] = v0 + c < V ? v[(size_t)(t0 + tt) * ld + (size_t)h * V + v0 + c] : 0.f;
            }
        }
        const int blocks = whole / BLK;
        for (int i = threadIdx.x; i < blocks * (COEF / 4); i += blockDim.x) {
            const int nb = i / (COEF / 4), c = (i % (COEF / 4)) * 4;
            copy16(sc + ((size_t)buf * NB + nb) * COEF + c, coef + ((size_t)(block0 + (t0 - begin) / BLK + nb) * H + h) * COEF + c);
        }
        if (whole > count) {  // a request's last block may hold fewer tokens: zeros in place of the missing ones
            for (int i = threadIdx.x; i < (whole - count) * RP; i += blockDim.x) {
                sq[((size_t)buf * TB + count) * RP + i] = 0.f;
                sk[((size_t)buf * TB + count) * RP + i] = 0.f;
            }
            for (int i = threadIdx.x; i < (whole - count) * COLS; i += blockDim.x) sv[((size_t)buf * TB + count) * COLS + i] = 0.f;
        }
        asm volatile("cp.async.commit_group;\n" ::);
    };

    // lanes of q and k beyond D are zeros in both buffers
    for (int i = threadIdx.x; i < 2 * TB * (DS - D); i += blockDim.x) {
        const int row = i / (DS - D), d = D + i % (DS - D);
        const int at = (d / DPT) * SEG + d % DPT;
        sq[(size_t)row * RP + at] = 0.f;
        sk[(size_t)row * RP + at] = 0.f;
    }
    fetch(begin, 0);
    for (int i = threadIdx.x; i < D * COLS; i += blockDim.x) {
        const int d = i / COLS, c = i % COLS;
        tile[d * (COLS + 1) + c] = v0 + c < V ? state[(size_t)d * V + v0 + c] : 0.f;
    }
    __syncthreads();
    float S[CPT][DPT];
#pragma unroll
    for (int c = 0; c < CPT; ++c)
#pragma unroll
        for (int i = 0; i < DPT; ++i) {
            const int d = sub * DPT + i;
            S[c][i] = d < D ? tile[d * (COLS + 1) + c0 + c] : 0.f;
        }
    const int live = max(0, min(CPT, V - (v0 + c0)));
    int buf = 0;
    for (int t0 = begin; t0 < end; t0 += TB, buf ^= 1) {
        asm volatile("cp.async.wait_group 0;\n" ::);
        __syncthreads();  // this stage has landed, and everybody has left the other buffer
        if (t0 + TB < end) fetch(t0 + TB, buf ^ 1);
        const int count = min(TB, end - t0);
        for (int tt = 0; tt < count; tt += BLK) {
            const float* bq = sq + ((size_t)buf * TB + tt) * RP + sub * SEG;
            const float* bk = sk + ((size_t)buf * TB + tt) * RP + sub * SEG;
            const float* bc = sc + ((size_t)buf * NB + tt / BLK) * COEF;
            // this thread's shares of S^T k and S^T q for the block's tokens
            float p[CPT][BLK], rd[CPT][BLK];
#pragma unroll
            for (int c = 0; c < CPT; ++c)
#pragma unroll
                for (int u = 0; u < BLK; ++u) p[c][u] = rd[c][u] = 0.f;
#pragma unroll
            for (int i = 0; i < DPT; i += 4)
#pragma unroll
                for (int u = 0; u < BLK; ++u) {
                    const float4 k4 = *reinterpret_cast<const float4*>(bk + u * RP + i), q4 = *reinterpret_cast<const float4*>(bq + u * RP + i);
                    const float kv[4] = {k4.x, k4.y, k4.z, k4.w}, qv[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
                    for (int c = 0; c < CPT; ++c)
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            p[c][u] = fmaf(S[c][i + e], kv[e], p[c][u]);
                            rd[c][u] = fmaf(S[c][i + e], qv[e], rd[c][u]);
                        }
                }
            float Mr[BLK], Pr[BLK], E[BLK];
#pragma unroll
            for (int i = 0; i < BLK; i += 4) {
                const float4 m4 = *reinterpret_cast<const float4*>(bc + sub * BLK + i), p4 = *reinterpret_cast<const float4*>(bc + 64 + sub * BLK + i),
                             e4 = *reinterpret_cast<const float4*>(bc + 136 + i);
                Mr[i] = m4.x; Mr[i + 1] = m4.y; Mr[i + 2] = m4.z; Mr[i + 3] = m4.w;
                Pr[i] = p4.x; Pr[i + 1] = p4.y; Pr[i + 2] = p4.z; Pr[i + 3] = p4.w;
                E[i] = e4.x; E[i + 1] = e4.y; E[i + 2] = e4.z; E[i + 3] = e4.w;
            }
            const float gt = bc[128 + sub], gl = bc[128 + BLK - 1];
            // from here lane `sub` stands for token tt + sub
            float w[CPT], o[CPT], un[CPT], ue[CPT][BLK];
#pragma unroll
            for (int c = 0; c < CPT; ++c) {
                w[c] = fmaf(-gt, trade_sum(p[c], sub), sv[((size_t)buf * TB + tt + sub) * COLS + c0 + c]);
                o[c] = gt * trade_sum(rd[c], sub);
                un[c] = 0.f;
            }
#pragma unroll
            for (int i = 0; i < BLK; ++i)
#pragma unroll
                for (int c = 0; c < CPT; ++c) un[c] = fmaf(Mr[i], __shfl_sync(0xffffffffu, w[c], i, TPC), un[c]);
#pragma unroll
            for (int i = 0; i < BLK; ++i)
#pragma unroll
                for (int c = 0; c < CPT; ++c) {
                    const float ui = __shfl_sync(0xffffffffu, un[c], i, TPC);
                    o[c] = fmaf(Pr[i], ui, o[c]);
                    ue[c][i] = ui * E[i];
                }
            if (tt + sub < count) {
                float* at = out + ((size_t)(t0 + tt + sub) * H + h) * V + v0 + c0;
                if (CPT == 4 && live == 4 && V % 4 == 0) *reinterpret_cast<float4*>(at) = make_float4(o[0], o[1 % CPT], o[2 % CPT], o[3 % CPT]);
                else
#pragma unroll
                    for (int c = 0; c < CPT; ++c)
                        if (c < live) at[c] = o[c];
            }
#pragma unroll
            for (int c = 0; c < CPT; ++c)
#pragma unroll
                for (int i = 0; i < DPT; ++i) S[c][i] *= gl;
#pragma unroll
            for (int i = 0; i < DPT; i += 4)
#pragma unroll
                for (int u = 0; u < BLK; ++u) {
                    const float4 k4 = *reinterpret_cast<const float4*>(bk + u * RP + i);
                    const float kv[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
                    for (int c = 0; c < CPT; ++c)
#pragma unroll
                        for (int e = 0; e < 4; ++e) S[c][i + e] = fmaf(kv[e], ue[c][u], S[c][i + e]);
                }
        }
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < CPT; ++c)
#pragma unroll
        for (int i = 0; i < DPT; ++i) {
            const int d = sub * DPT + i;
            if (d < D) tile[d * (COLS + 1) + c0 + c] = S[c][i];
        }
    __syncthreads();
    for (int i = threadIdx.x; i < D * COLS; i += blockDim.x) {
        const int d = i / COLS, c = i % COLS;
        if (v0 + c < V) state[(size_t)d * V + v0 + c] = tile[d * (COLS + 1) + c];
    }
}

// Few tokens a request.  grid (H, requests); Vp (V rounded up to whole warps) * parts threads: thread (part, column) holds rows
// part * DPT ... of its column.  y: rows [q: G*D | k: G*D | v: H*V] before the unit norms.  gate: [N, H * V] (pitch ldg).
// out[t, h*V + c] = rms_norm over the head (o) * weight * silu(gate)
template <int DPT, typename TO>
__global__ void __launch_bounds__(512)
delta_step_kernel(const float* __restrict__ y, int ldy, const float* __restrict__ b, int ldb, const float* __restrict__ a, int lda,
                  const float* __restrict__ a_log, const float* __restrict__ dt_bias, const float* __restrict__ gate, int ldg,
                  const float* __restrict__ weight, float* __restrict__ states, const int* __restrict__ state_slots,
                  const int* __restrict__ cu_tokens, TO* __restrict__ out, int ldo, int H, int G, int D, int V, int Vp, int parts,
                  float q_scale, float eps) {
    extern __shared__ __align__(16) float shared[];
    const int DS = DPT * parts;
    float* sk = shared;                    // [DS]
    float* sq = sk + DS;                   // [DS]
    float* red = sq + DS;                  // [parts][2][Vp]
    float* scratch = red + 2 * parts * Vp; // [32]
    pdl_trigger();
    const int h = blockIdx.x, r = blockIdx.y, g = h / (H / G);
    const int c = threadIdx.x % Vp, part = threadIdx.x / Vp, lane = threadIdx.x & 31;
    const int begin = cu_tokens[r], end = cu_tokens[r + 1], slot = state_slots[r];
    float* state = states + ((size_t)slot * H + h) * D * V;
    const float al = a_log[h], db = dt_bias[h], wt = c < V ? weight[c] : 0.f;
    pdl_wait();
    float S[DPT];
#pragma unroll
    for (int i = 0; i < DPT; ++i) {
        const int d = part * DPT + i;
        S[i] = c < V && d < D ? state[(size_t)d * V + c] : 0.f;
    }
    for (int t = begin; t < end; ++t) {
        const float* row = y + (size_t)t * ldy;
        const float vt = c < V ? row[(size_t)2 * G * D + (size_t)h * V + c] : 0.f;
        const float zt = c < V ? gate[(size_t)t * ldg + (size_t)h * V + c] : 0.f;
        const float gt = expf(log_decay(a[(size_t)t * lda + h], db, al)), beta = sigmoid_of(b[(size_t)t * ldb + h]);
        for (int d = threadIdx.x; d < DS; d += blockDim.x) {
            sq[d] = d < D ? row[(size_t)g * D + d] : 0.f;
            sk[d] = d < D ? row[(size_t)(G + g) * D + d] : 0.f;
        }
        __syncthreads();
        // every warp sums up the whole vectors by itself, in the same order
        float qq = 0.f, kk = 0.f, kq = 0.f;
        for (int d = lane; d < DS; d += 32) {
            const float qv = sq[d], kv = sk[d];
            qq = fmaf(qv, qv, qq);
            kk = fmaf(kv, kv, kk);
            kq = fmaf(kv, qv, kq);
        }
        const float fq = q_scale / sqrtf(warp_sum(qq) + 1e-6f), fk = 1.f / sqrtf(warp_sum(kk) + 1e-6f);
        kq = warp_sum(kq) * fq * fk;
        float p = 0.f, rd = 0.f;
#pragma unroll
        for (int i = 0; i < DPT; ++i) {
            p = fmaf(S[i], sk[part * DPT + i], p);
            rd = fmaf(S[i], sq[part * DPT + i], rd);
        }
        red[(part * 2) * Vp + c] = p;
        red[(part * 2 + 1) * Vp + c] = rd;
        __syncthreads();
        p = rd = 0.f;
        for (int i = 0; i < parts; ++i) {
            p += red[(i * 2) * Vp + c];
            rd += red[(i * 2 + 1) * Vp + c];
        }
        const float u = beta * (vt - gt * fk * p);
        const float o = c < V ? fmaf(kq, u, gt * fq * rd) : 0.f;
        const float uk = u * fk;
#pragma unroll
        for (int i = 0; i < DPT; ++i) S[i] = fmaf(sk[part * DPT + i], uk, gt * S[i]);
        const float ss = warp_sum(o * o);
        if (part == 0 && lane == 0) scratch[c >> 5] = ss;
        __syncthreads();
        if (part == 0 && c < V) {
            float total = 0.f;
            for (int i = 0; i < (Vp >> 5); ++i) total += scratch[i];
            const float n = o / sqrtf(total / (float)V + eps) * wt * (zt * sigmoid_of(zt));
            out[(size_t)t * ldo + (size_t)h * V + c] = from_float<TO>(n);
        }
    }
#pragma unroll
    for (int i = 0; i < DPT; ++i) {
        const int d = part * DPT + i;
        if (c < V && d < D) state[(size_t)d * V + c] = S[i];
    }
}

template <typename K>
int room(K kernel, size_t smem) {
    if (smem <= 48 * 1024) return 0;
    return (int)cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
}

}  // namespace

// The way for prompts, two launches.  y: [N, >= 2*G*D + H*V] float32 (q and k are left as unit vectors); b, a: [N, H] float32;
// coef: room for (N / 8 + requests + 1) * H * 144 floats; out: [N, H, V] float32.  wide_columns: 0 = 16 columns of the state a
// CTA, 1 = as many as the registers take (steps with CTAs enough).
LLM_EXPORT int llm_delta_scan(float* y, int ldy, const float* b, int ldb, const float* a, int lda, const float* a_log, const float* dt_bias,
                              float* states, const int* state_slots, const int* cu_tokens, float* coef, float* out, int requests,
                              int max_query_len, int G, int H, int D, int V, float q_scale, int wide_columns, cudaStream_t stream) {
    if (requests <= 0 || max_query_len <= 0) return 0;
    if (G <= 0 || H <= 0 || H % G || H > 65535 || D <= 0 || D > 256 || V <= 0 || requests > 65535 || ldy < 2 * G * D + H * V || !coef) return LLM_ERR_BAD_ARGUMENT;
    const int D4 = (D + 3) & ~3;
    const size_t psmem = (size_t)2 * BLK * (D4 + 4) * sizeof(float);
    int code = launch_pdl(delta_prepare_kernel, dim3((max_query_len + BLK - 1) / BLK, G, requests), dim3(128), psmem, stream, y, ldy, b, ldb, a, lda, a_log,
                          dt_bias, cu_tokens, coef, G, H, D, q_scale);
    if (code != 0) return code;
    const float *q = y, *k = y + (size_t)G * D, *v = y + (size_t)2 * G * D;
    auto go = [&](auto kernel, int dpt, int tb, int cpt) -> int {
        const int cols = GROUPS * cpt, ds = dpt * TPC;
        const size_t smem = ((size_t)4 * tb * (dpt + 4) * TPC + (size_t)2 * tb * cols + (size_t)2 * (tb / BLK) * COEF + (size_t)ds * (cols + 1)) * sizeof(float);
        const int e = room(kernel, smem);
        if (e != 0) return e;
        return launch_pdl(kernel, dim3((V + cols - 1) / cols, H, requests), dim3(GROUPS * TPC), smem, stream, q, k, v, ldy, (const float*)coef, states,
                          state_slots, cu_tokens, out, H, G, D, V);
    };
    if (D <= 32) return wide_columns ? go(delta_scan_kernel<4, 32, 4>, 4, 32, 4) : go(delta_scan_kernel<4, 32, 1>, 4, 32, 1);
    if (D <= 64) return wide_columns ? go(delta_scan_kernel<8, 32, 4>, 8, 32, 4) : go(delta_scan_kernel<8, 32, 1>, 8, 32, 1);
    if (D <= 128) return wide_columns ? go(delta_scan_kernel<16, 16, 2>, 16, 16, 2) : go(delta_scan_kernel<16, 16, 1>, 16, 16, 1);
    return go(delta_scan_kernel<32, 16, 1>, 32, 16, 1);
}

// The way for few tokens a request, one launch: the recurrence, the norm over each head, its weight [V] and the gate.
// LLM_ERR_UNSUPPORTED where a head's state does not fit a CTA's registers.
LLM_EXPORT int llm_delta_step(const float* y, int ldy, const float* b, int ldb, const float* a, int lda, const float* a_log, const float* dt_bias,
                              const float* gate, int ldg, const float* weight, float* states, const int* state_slots, const int* cu_tokens,
                              void* out, int out_dtype, int ldo, int requests, int G, int H, int D, int V, float q_scale, float eps,
                              cudaStream_t stream) {
    if (requests <= 0) return 0;
    if (G <= 0 || H <= 0 || H % G || D <= 0 || V <= 0 || requests > 65535 || ldy < 2 * G * D + H * V || ldg < H * V || ldo < H * V) return LLM_ERR_BAD_ARGUMENT;
    const int Vp = (V + 31) / 32 * 32;
    int dpt = 8;
    while (dpt < 32 && (D + dpt - 1) / dpt * Vp > 512) dpt *= 2;
    const int parts = (D + dpt - 1) / dpt;
    if (parts * Vp > 512) return LLM_ERR_UNSUPPORTED;
    const size_t smem = ((size_t)2 * dpt * parts + (size_t)2 * parts * Vp + 32) * sizeof(float);
    auto go = [&](auto kernel, auto* op) -> int {
        return launch_pdl(kernel, dim3(H, requests), dim3(parts * Vp), smem, stream, y, ldy, b, ldb, a, lda, a_log, dt_bias, gate, ldg, weight, states,
                          state_slots, cu_tokens, op, ldo, H, G, D, V, Vp, parts, q_scale, eps);
    };
    using bf = __nv_bfloat16;
    if (out_dtype == LLM_F32)
        return dpt == 8 ? go(delta_step_kernel<8, float>, (float*)out) : dpt == 16 ? go(delta_step_kernel<16, float>, (float*)out) : go(delta_step_kernel<32, float>, (float*)out);
    if (out_dtype == LLM_BF16)
        return dpt == 8 ? go(delta_step_kernel<8, bf>, (bf*)out) : dpt == 16 ? go(delta_step_kernel<16, bf>, (bf*)out) : go(delta_step_kernel<32, bf>, (bf*)out);
    return LLM_ERR_BAD_ARGUMENT;
}
