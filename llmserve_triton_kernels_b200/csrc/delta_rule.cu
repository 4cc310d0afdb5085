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
// The unit vectors lie in memory as the walk reads them: two tokens' lanes next to one another, so that one packed multiply-add
// (fma.rn.f32x2) serves two tokens, and a block's vectors in one run.
#include "common.cuh"

namespace {

constexpr int BLK = 8;     // tokens a block
constexpr int COEF = 144;  // floats a (block, head): M [8][8], P [8][8], G [8], E [8]
constexpr int R = 16;      // lanes of the scan that share a group of columns of the state: each holds D / 16 rows of them
constexpr int THREADS = 128;

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

// Two tokens at once: a.x * b.x + c.x and a.y * b.y + c.y, each as fmaf would give it.
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
    float2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(reinterpret_cast<unsigned long long&>(d)) : "l"(reinterpret_cast<unsigned long long&>(a)),
        "l"(reinterpret_cast<unsigned long long&>(b)), "l"(reinterpret_cast<unsigned long long&>(c)));
    return d;
}

__device__ __forceinline__ float2 mul2(float2 a, float2 b) {
    float2 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(reinterpret_cast<unsigned long long&>(d)) : "l"(reinterpret_cast<unsigned long long&>(a)),
        "l"(reinterpret_cast<unsigned long long&>(b)));
    return d;
}

// grid (blocks of the longest request, G, requests), 128 threads.  y: rows [q: G*D | k: G*D | ...] (pitch ldy).
// units: [blocks, G, 2 (k, q), 4 (pairs of tokens), DS, 2], zeros for missing tokens and for lanes from D on.  coef: [blocks, H, COEF]
__global__ void __launch_bounds__(128)
delta_prepare_kernel(const float* __restrict__ y, int ldy, const float* __restrict__ b, int ldb, const float* __restrict__ a, int lda,
                     const float* __restrict__ a_log, const float* __restrict__ dt_bias, const int* __restrict__ cu_tokens,
                     float* __restrict__ units, float* __restrict__ coef, int G, int H, int D, int DS, float q_scale) {
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
    const size_t block = first_block(request, r) + blockIdx.x;
    pdl_wait();
    {
        const int t = warp * 2;  // a warp has a pair of tokens
        const bool has0 = t < count, has1 = t + 1 < count;
        const float *q0 = y + (size_t)(begin + t) * ldy + (size_t)g * D, *q1 = q0 + ldy, *k0 = q0 + (size_t)G * D, *k1 = q1 + (size_t)G * D;
        float s[4] = {0.f, 0.f, 0.f, 0.f};
        for (int d = lane; d < D4; d += 32) {
            const float v[4] = {has0 && d < D ? q0[d] : 0.f, has1 && d < D ? q1[d] : 0.f, has0 && d < D ? k0[d] : 0.f, has1 && d < D ? k1[d] : 0.f};
#pragma unroll
            for (int e = 0; e < 4; ++e) s[e] = fmaf(v[e], v[e], s[e]);
            sq[t * pitch + d] = v[0];
            sq[(t + 1) * pitch + d] = v[1];
            sk[t * pitch + d] = v[2];
            sk[(t + 1) * pitch + d] = v[3];
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) s[e] = (e < 2 ? q_scale : 1.f) / sqrtf(warp_sum(s[e]) + 1e-6f);
        float2* uk = reinterpret_cast<float2*>(units + ((block * G + g) * 2 * 4 + warp) * DS * 2);
        float2* uq = uk + (size_t)4 * DS;
        for (int d = lane; d < DS; d += 32) {
            float2 qv = make_float2(0.f, 0.f), kv = qv;
            if (d < D4) {
                qv = make_float2(sq[t * pitch + d] * s[0], sq[(t + 1) * pitch + d] * s[1]);
                kv = make_float2(sk[t * pitch + d] * s[2], sk[(t + 1) * pitch + d] * s[3]);
                sq[t * pitch + d] = qv.x;
                sq[(t + 1) * pitch + d] = qv.y;
                sk[t * pitch + d] = kv.x;
                sk[(t + 1) * pitch + d] = kv.y;
            }
            uk[d] = kv;
            uq[d] = qv;
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
        float* to = coef + (block * H + h) * COEF;
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

// Sixteen lanes hold partial sums of two columns for eight tokens; they trade halves (columns, then tokens) so that lane `sub` ends
// with the sum of column sub / 8 for token sub % 8.  Every lane has its sums in an order of its own, in which what it keeps stands in
// front: x[0] is its own column, x[c][u] the pair of tokens u ^ (sub % 8 / 2); so nothing is selected on the way but the last half.
__device__ __forceinline__ float trade_sum(const float2 (&x)[2][BLK / 2], int sub) {
    float2 a[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
        a[u].x = x[0][u].x + __shfl_xor_sync(0xffffffffu, x[1][u].x, 8);
        a[u].y = x[0][u].y + __shfl_xor_sync(0xffffffffu, x[1][u].y, 8);
    }
#pragma unroll
    for (int u = 0; u < 2; ++u) {
        a[u].x += __shfl_xor_sync(0xffffffffu, a[u + 2].x, 4);
        a[u].y += __shfl_xor_sync(0xffffffffu, a[u + 2].y, 4);
    }
    a[0].x += __shfl_xor_sync(0xffffffffu, a[1].x, 2);
    a[0].y += __shfl_xor_sync(0xffffffffu, a[1].y, 2);
    return (sub & 1 ? a[0].y : a[0].x) + __shfl_xor_sync(0xffffffffu, sub & 1 ? a[0].x : a[0].y, 1);
}

// grid (columns of V, H, requests), 128 threads: 8 groups of 16 lanes; a group owns 2 * MC neighbouring columns, a lane DPT rows of
// them: rows 2 (j * 16 + lane) and the one behind for j < DPT / 2.  Of two neighbouring columns a lane has its own (lane / 8) first,
// and it takes the block's pairs of tokens in the order u ^ (lane % 8 / 2) (see trade_sum).  units, coef: as above (DS = 16 * DPT); v: [N, H * V] (pitch ld);
// out: [N, H, V] float32.  NB blocks a stage, the next stage on its way (cp.async) while one is walked.
template <int DPT, int NB, int MC>
__global__ void __launch_bounds__(THREADS)
delta_scan_kernel(const float* __restrict__ units, const float* __restrict__ v, int ld, const float* __restrict__ coef, float* __restrict__ states,
                  const int* __restrict__ state_slots, const int* __restrict__ cu_tokens, float* __restrict__ out, int H, int G, int D, int V) {
    constexpr int CPT = 2 * MC, COLS = THREADS / R * CPT, DS = R * DPT, TB = NB * BLK, J = DPT / 2;
    constexpr int UNITS = 2 * BLK * DS;    // floats a block: k, then q
    constexpr bool KEEP = DPT <= 8;        // a lane's share of the block's k stays in registers from the dots to the update
    extern __shared__ __align__(16) float shared[];
    float* su = shared;                    // [2][NB][UNITS]
    float* sc = su + 2 * NB * UNITS;       // [2][NB][COEF]
    float* sv = sc + 2 * NB * COEF;        // [2][TB][COLS]
    float* tile = su;                      // [DS][COLS + 1], the state on its way in and out (before the first and after the last stage)
    pdl_trigger();
    const int r = blockIdx.z, h = blockIdx.y, v0 = blockIdx.x * COLS, g = h / (H / G);
    const int sub = threadIdx.x % R, c0 = (threadIdx.x / R) * CPT;
    const int col = sub >> 3, tok = sub & 7, turn = tok >> 1;  // what this lane stands for between the sums, and its order of pairs
    const int begin = cu_tokens[r], end = cu_tokens[r + 1], slot = state_slots[r];
    const size_t block0 = first_block(begin, r);
    float* state = states + ((size_t)slot * H + h) * D * V;
    const bool vec_v = V % 4 == 0 && ld % 4 == 0 && reinterpret_cast<uintptr_t>(v) % 16 == 0 && v0 + COLS <= V;
    pdl_wait();
    if (begin >= end) return;

    for (int i = threadIdx.x; i < D * COLS; i += THREADS) {
        const int d = i / COLS, c = i % COLS;
        tile[d * (COLS + 1) + c] = v0 + c < V ? state[(size_t)d * V + v0 + c] : 0.f;
    }
    __syncthreads();
    float S[CPT][J][2];
#pragma unroll
    for (int c = 0; c < CPT; ++c)
#pragma unroll
        for (int j = 0; j < J; ++j)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int d = 2 * (j * R + sub) + e;
                S[c][j][e] = d < D ? tile[d * (COLS + 1) + c0 + (c ^ col)] : 0.f;
            }
    __syncthreads();

    auto fetch = [&](int t0, int buf) {
        const int count = min(TB, end - t0), blocks = (count + BLK - 1) / BLK;
        const size_t at = block0 + (t0 - begin) / BLK;
#pragma unroll
        for (int nb = 0; nb < NB; ++nb) {
            if (nb >= blocks) break;
            const float* from = units + ((at + nb) * G + g) * UNITS;
            float* to = su + (size_t)(buf * NB + nb) * UNITS;
#pragma unroll
            for (int i = 0; i < UNITS / 4; i += THREADS)
                if (UNITS / 4 % THREADS == 0 || i + (int)threadIdx.x < UNITS / 4) copy16(to + (i + threadIdx.x) * 4, from + (i + threadIdx.x) * 4);
            if (threadIdx.x < COEF / 4) copy16(sc + (size_t)(buf * NB + nb) * COEF + threadIdx.x * 4, coef + ((at + nb) * H + h) * COEF + threadIdx.x * 4);
        }
        if (vec_v) {
            for (int i = threadIdx.x; i < count * (COLS / 4); i += THREADS) {
                const int tt = i / (COLS / 4), c = (i % (COLS / 4)) * 4;
                copy16(sv + ((size_t)buf * TB + tt) * COLS + c, v + (size_t)(t0 + tt) * ld + (size_t)h * V + v0 + c);
            }
        } else {
            for (int i = threadIdx.x; i < count * COLS; i += THREADS) {
                const int tt = i / COLS, c = i % COLS;
                sv[((size_t)buf * TB + tt) * COLS + c] = v0 + c < V ? v[(size_t)(t0 + tt) * ld + (size_t)h * V + v0 + c] : 0.f;
            }
        }
        for (int i = threadIdx.x; i < (blocks * BLK - count) * COLS; i += THREADS) sv[((size_t)buf * TB + count) * COLS + i] = 0.f;
        asm volatile("cp.async.commit_group;\n" ::);
    };

    fetch(begin, 0);
    int buf = 0;
    for (int t0 = begin; t0 < end; t0 += TB, buf ^= 1) {
        asm volatile("cp.async.wait_group 0;\n" ::);
        __syncthreads();  // this stage has landed, and everybody has left the other buffer
        if (t0 + TB < end) fetch(t0 + TB, buf ^ 1);
        const int count = min(TB, end - t0);
#pragma unroll 1
        for (int nb = 0; nb * BLK < count; ++nb) {
            const float4* bk = reinterpret_cast<const float4*>(su + (size_t)(buf * NB + nb) * UNITS) + sub;
            const float4* bq = bk + BLK * DS / 4;
            const float* bc = sc + (size_t)(buf * NB + nb) * COEF;
            // this lane's shares of S^T k and S^T q for the block's tokens, two tokens a packed sum
            float2 p[MC][2][BLK / 2], rd[MC][2][BLK / 2], kk[KEEP ? J : 1][BLK / 2][2];
#pragma unroll
            for (int j = 0; j < J; ++j) {
                float2 ss[CPT][2];
#pragma unroll
                for (int c = 0; c < CPT; ++c)
#pragma unroll
                    for (int e = 0; e < 2; ++e) ss[c][e] = make_float2(S[c][j][e], S[c][j][e]);
#pragma unroll
                for (int u = 0; u < BLK / 2; ++u) {
                    // rows 2 (j R + sub), + 1 of tokens 2 (u ^ turn), + 1
                    const float4 k4 = bk[(u ^ turn) * (DS / 2) + j * R], q4 = bq[(u ^ turn) * (DS / 2) + j * R];
                    const float2 k2[2] = {make_float2(k4.x, k4.y), make_float2(k4.z, k4.w)}, q2[2] = {make_float2(q4.x, q4.y), make_float2(q4.z, q4.w)};
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        if (KEEP) kk[j][u][e] = k2[e];
#pragma unroll
                        for (int c = 0; c < CPT; ++c) {
                            float2 &pc = p[c / 2][c % 2][u], &rc = rd[c / 2][c % 2][u];
                            pc = j == 0 && e == 0 ? mul2(ss[c][e], k2[e]) : fma2(ss[c][e], k2[e], pc);
                            rc = j == 0 && e == 0 ? mul2(ss[c][e], q2[e]) : fma2(ss[c][e], q2[e], rc);
                        }
                    }
                }
            }
            float Mr[BLK];
            float2 Pr[BLK / 2], E[BLK / 2];  // in the lane's order of pairs
#pragma unroll
            for (int i = 0; i < BLK; i += 4) {
                const float4 m4 = *reinterpret_cast<const float4*>(bc + tok * BLK + i);
                Mr[i] = m4.x; Mr[i + 1] = m4.y; Mr[i + 2] = m4.z; Mr[i + 3] = m4.w;
            }
#pragma unroll
            for (int u = 0; u < BLK / 2; ++u) {
                Pr[u] = *reinterpret_cast<const float2*>(bc + 64 + tok * BLK + 2 * (u ^ turn));
                E[u] = *reinterpret_cast<const float2*>(bc + 136 + 2 * (u ^ turn));
            }
            const float gt = bc[128 + tok], gl = bc[128 + BLK - 1];
            float w[MC], o[MC], un[MC];
            float2 ue[CPT][BLK / 2];
#pragma unroll
            for (int m = 0; m < MC; ++m) {
                w[m] = fmaf(-gt, trade_sum(p[m], sub), sv[((size_t)buf * TB + nb * BLK + tok) * COLS + c0 + 2 * m + col]);
                float even = 0.f, odd = 0.f;
#pragma unroll
                for (int i = 0; i < BLK; i += 2) {
                    even = fmaf(Mr[i], __shfl_sync(0xffffffffu, w[m], i, 8), even);
                    odd = fmaf(Mr[i + 1], __shfl_sync(0xffffffffu, w[m], i + 1, 8), odd);
                }
                un[m] = even + odd;
            }
#pragma unroll
            for (int m = 0; m < MC; ++m) o[m] = gt * trade_sum(rd[m], sub);
#pragma unroll
            for (int u = 0; u < BLK / 2; ++u) {
                const int from = 2 * (u ^ turn) + (sub & 8);
#pragma unroll
                for (int m = 0; m < MC; ++m) {
                    const float2 mine = make_float2(__shfl_sync(0xffffffffu, un[m], from, 16), __shfl_sync(0xffffffffu, un[m], from + 1, 16));
                    const float2 other = make_float2(__shfl_sync(0xffffffffu, un[m], from ^ 8, 16), __shfl_sync(0xffffffffu, un[m], (from ^ 8) + 1, 16));
                    o[m] = fmaf(Pr[u].x, mine.x, o[m]);
                    o[m] = fmaf(Pr[u].y, mine.y, o[m]);
                    ue[2 * m][u] = mul2(mine, E[u]);
                    ue[2 * m + 1][u] = mul2(other, E[u]);
                }
            }
            if (nb * BLK + tok < count) {
#pragma unroll
                for (int m = 0; m < MC; ++m)
                    if (v0 + c0 + 2 * m + col < V) out[((size_t)(t0 + nb * BLK + tok) * H + h) * V + v0 + c0 + 2 * m + col] = o[m];
            }
#pragma unroll
            for (int j = 0; j < J; ++j) {
                float2 k2[BLK / 2][2];
#pragma unroll
                for (int u = 0; u < BLK / 2; ++u) {
                    if (KEEP) { k2[u][0] = kk[j][u][0]; k2[u][1] = kk[j][u][1]; }
                    else {
                        const float4 k4 = bk[(u ^ turn) * (DS / 2) + j * R];
                        k2[u][0] = make_float2(k4.x, k4.y);
                        k2[u][1] = make_float2(k4.z, k4.w);
                    }
                }
#pragma unroll
                for (int c = 0; c < CPT; ++c)
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        float2 acc = mul2(k2[0][e], ue[c][0]);
#pragma unroll
                        for (int u = 1; u < BLK / 2; ++u) acc = fma2(k2[u][e], ue[c][u], acc);
                        S[c][j][e] = fmaf(gl, S[c][j][e], acc.x) + acc.y;
                    }
            }
        }
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < CPT; ++c)
#pragma unroll
        for (int j = 0; j < J; ++j)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int d = 2 * (j * R + sub) + e;
                if (d < D) tile[d * (COLS + 1) + c0 + (c ^ col)] = S[c][j][e];
            }
    __syncthreads();
    for (int i = threadIdx.x; i < D * COLS; i += THREADS) {
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

// Rows of a head's q or k as the scan has them in memory and in registers: 16 lanes of 2, 4, 8 or 16 rows.
LLM_EXPORT int llm_delta_rows(int D) { return D <= 32 ? 32 : D <= 64 ? 64 : D <= 128 ? 128 : 256; }

// The way for prompts, two launches.  y: [N, >= 2*G*D + H*V] float32; b, a: [N, H] float32; scratch: room for N / 8 + requests + 1
// blocks of G * 16 * llm_delta_rows(D) + H * 144 floats; out: [N, H, V] float32.  sms: SMs of the device.
LLM_EXPORT int llm_delta_scan(const float* y, int ldy, const float* b, int ldb, const float* a, int lda, const float* a_log, const float* dt_bias,
                              float* states, const int* state_slots, const int* cu_tokens, float* scratch, float* out, int N, int requests,
                              int max_query_len, int G, int H, int D, int V, float q_scale, int sms, cudaStream_t stream) {
    if (requests <= 0 || max_query_len <= 0) return 0;
    if (G <= 0 || H <= 0 || H % G || H > 65535 || D <= 0 || D > 256 || V <= 0 || requests > 65535 || ldy < 2 * G * D + H * V || !scratch || sms <= 0)
        return LLM_ERR_BAD_ARGUMENT;
    const int D4 = (D + 3) & ~3, DS = llm_delta_rows(D);
    float* units = scratch;
    float* coef = scratch + (size_t)(N / BLK + requests + 1) * G * 2 * BLK * DS;
    const size_t psmem = (size_t)2 * BLK * (D4 + 4) * sizeof(float);
    int code = launch_pdl(delta_prepare_kernel, dim3((max_query_len + BLK - 1) / BLK, G, requests), dim3(128), psmem, stream, y, ldy, b, ldb, a, lda, a_log,
                          dt_bias, cu_tokens, units, coef, G, H, D, DS, q_scale);
    if (code != 0) return code;
    const float* v = y + (size_t)2 * G * D;
    auto go = [&](auto kernel, int nb, int mc) -> int {
        const int cols = THREADS / R * 2 * mc;
        const dim3 grid((V + cols - 1) / cols, H, requests);
        size_t smem = ((size_t)2 * nb * (2 * BLK * DS + COEF) + (size_t)2 * nb * BLK * cols) * sizeof(float);
        const size_t tile = (size_t)DS * (cols + 1) * sizeof(float);
        if (tile > smem) smem = tile;
        // A CTA lives as long as the request.  It starts while the last CTAs of the kernel in front still stand on most SMs, and would
        // crowd onto those that are free first: with few CTAs, each asks for so much shared memory that they spread out evenly.
        const long long ctas = (long long)grid.x * grid.y * grid.z;
        for (int per = 1; per <= 3; ++per)
            if (ctas <= (long long)per * sms) {
                const size_t want = (size_t)(227 * 1024) / (per + 1) + 1024;
                if (want > smem) smem = want;
                break;
            }
        const int e = room(kernel, smem);
        if (e != 0) return e;
        return launch_pdl(kernel, grid, dim3(THREADS), smem, stream, (const float*)units, v, ldy, (const float*)coef, states, state_slots, cu_tokens, out,
                          H, G, D, V);
    };
    const bool wide = (long long)((V + 31) / 32) * H * requests >= 2LL * sms;  // CTAs enough when each takes 32 columns of the state
    if (DS == 32) return wide ? go(delta_scan_kernel<2, 4, 2>, 4, 2) : go(delta_scan_kernel<2, 4, 1>, 4, 1);
    if (DS == 64) return wide ? go(delta_scan_kernel<4, 4, 2>, 4, 2) : go(delta_scan_kernel<4, 4, 1>, 4, 1);
    if (DS == 128) return wide ? go(delta_scan_kernel<8, 2, 2>, 2, 2) : go(delta_scan_kernel<8, 2, 1>, 2, 1);
    return go(delta_scan_kernel<16, 2, 1>, 2, 1);
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
