// Causal (optionally windowed) grouped-query attention over the paged cache for prompt portions, on the
// fifth-generation tensor cores: both products of a key tile (scores = Q K^T, output += P V) are
// tcgen05.mma with their accumulators AND their A operands (queries, probabilities) in tensor memory; keys and
// values come into shared memory by TMA (128-byte swizzle), page by page through the request's page table.
//
// One CTA computes 128 query tokens of one head against the keys they may see, 64 keys at a time:
//   warps 0-3 : softmax.  Thread i owns query row i, which is lane i of tensor memory: it puts its queries there
//               once, reads its 64 scores with tcgen05.ld, keeps the running maximum and sum of the row (no
//               shuffles: the whole row is the thread's) and stores the probabilities as bfloat16 into its lane,
//               where the second product reads them.  The output accumulates in tensor memory over all key
//               tiles; a row's shift follows its maximum only when the maximum has risen by more than 2^8, and
//               only then does the warp rescale its 32 rows of the output (load, multiply, store).
//   warps 4, 6: producers of keys and of values.  Each looks up pages (32 entries of the page table per load,
//               handed round by shuffles) and issues one TMA box per page, each from a lane of its own, into
//               rings of STAGES tiles; a stage of keys is free as soon as its scores are computed.
//   warps 5, 7: one thread of each issues a product (5 the scores, 7 the output); warp 5 owns the allocation of
//               tensor memory.
// Scores have two buffers: those of tile j+1 are computed while the softmax of tile j runs, and the second
// product of tile j runs while the softmax of tile j+1 does.  Two CTAs share an SM.  Softmax, running sums and
// the output are 32-bit; probabilities are rounded to bfloat16 for the second product, as in the mma.sync kernel.
//
// Keys past a request's length inside its last page, and pages outside the range a CTA needs, are
// never looked at: a score outside [window start, position] is -inf before the exponential, and the
// producer loads a page of the needed range in place of one outside it, so that no stale or released
// page is touched.  Values of masked keys meet a probability of exactly zero; the cache pool holds only
// finite numbers (it starts as zeros and is written by the projection kernels).
//
// Every mbarrier wait is bounded; a wait that gives up sets *error_flag, the roles leave their loops,
// tensor memory is freed and the kernel returns.
#include "attention_tile.cuh"
#ifdef ATT_PROF
#include <cstdio>
#endif
#include "umma.cuh"

namespace {

using attn::AttnParams;

constexpr int BM = 128, BN = 64, THREADS = 256, TMEM_COLS = 256;
constexpr float LAZY = 8.f;  // log2 of how far a row's maximum may rise before its shift follows

// What differs between the sizes of a head: KD lanes of a query and a key, VD of a value.  256 columns of tensor memory a CTA (two CTAs share an SM's 512), two
// bfloat16 to a column where an A operand lies:
//   head size 64 : two tiles of scores [0, 64), [64, 128); the output [128, 192); the queries [192, 224); a tile's
//                  probabilities [224, 256).  Three stages of keys and of values (16 KB a stage): 49 KB of shared memory.
//   head size 128: one tile of scores [0, 64); the output [64, 192); probabilities [192, 224).  The queries do not fit
//                  and stay in shared memory (32 KB, the first product's A operand from there); two stages of keys
//                  and of values (32 KB a stage): 97 KB.  With one buffer of scores the product of tile j+1 starts when
//                  the softmax has read tile j; the other CTA of the SM fills the gap.
//   64 and 128   : one tile of scores [0, 64); the output [64, 192); the queries [192, 224); probabilities [224, 256).  Three stages
//                  (24 KB): 73 KB.
template <int KD, int VD>
struct Shape {
    static constexpr bool Q_IN_TMEM = KD == 64;
    static constexpr int S_BUFFERS = VD == 64 ? 2 : 1, STAGES = KD == 64 ? 3 : 2;
    static constexpr int O_COL = S_BUFFERS * BN, Q_COL = O_COL + VD, P_COL = Q_IN_TMEM ? Q_COL + KD / 2 : O_COL + VD;
    static constexpr int K_HALVES = KD / 64, V_HALVES = VD / 64;  // 64-wide pieces of a row of keys (queries), values: one TMA box each
    static constexpr int K_BYTES = BN * KD * 2, V_BYTES = BN * VD * 2, STAGE_BYTES = K_BYTES + V_BYTES, Q_BYTES = Q_IN_TMEM ? 0 : BM * KD * 2;
    static constexpr size_t SMEM = 1024 + (size_t)Q_BYTES + (size_t)STAGES * STAGE_BYTES;
    static_assert(P_COL + BN / 2 <= TMEM_COLS, "tensor memory");
};

struct TcParams {
    AttnParams a;
    int min_tokens;         // requests with fewer tokens are other kernels'
    int tiles_per_request;  // 128-token tiles of the longest request
    int* error_flag;
    // Heads of several score maps: blockIdx.x counts (head, map), the queries of a head's maps lie side by side, its keys' likewise
    // in a row of the pool (map m from lane m * KD on), all maps over the same values.
    int maps;
    // The result of every (token, head, map) as it is, 32-bit [tokens, H * maps, VD], for a kernel that joins the maps; null: bfloat16 to a.out
    float* raw;
    // The values were cached turned by their positions' angles: lanes m and m + VD/2 of the result are turned back by the query
    // token's row of (cos, sin) [tokens, VD / 2]; null: not
    const float2* turn;
    // One gate a head: the result times sigmoid(gate[token * gate_token + head]); null: none
    const float* gate;
    long long gate_token;
};

__device__ __forceinline__ void mbar_arrive(unsigned long long* bar) { tma::mbar_arrive(bar); }

template <int KD, int VD>
__global__ void __launch_bounds__(THREADS, 2)
attention_tcgen05_kernel(const TcParams tp, const __grid_constant__ CUtensorMap qmap, const __grid_constant__ CUtensorMap kvmap) {
    using Sh = Shape<KD, VD>;
    constexpr int STAGES = Sh::STAGES, NBUF = Sh::S_BUFFERS, K_BYTES = Sh::K_BYTES, STAGE_BYTES = Sh::STAGE_BYTES;
    constexpr int K_HALVES = Sh::K_HALVES, V_HALVES = Sh::V_HALVES;
    constexpr int O_COL = Sh::O_COL, Q_COL = Sh::Q_COL, P_COL = Sh::P_COL;
    const AttnParams& p = tp.a;
    const int q_head = blockIdx.x, head = q_head / tp.maps, kvh = head / p.G;
    const int r = blockIdx.y / tp.tiles_per_request;
    const int tile = tp.tiles_per_request - 1 - (int)(blockIdx.y % tp.tiles_per_request);  // long tiles first
    const int q_begin = p.cu_tokens[r], q_len = p.cu_tokens[r + 1] - q_begin;
    if (q_len < tp.min_tokens) return;
    const int row0 = tile * BM;
    if (row0 >= q_len) return;
    const int rows_here = min(BM, q_len - row0);
    const int pos0 = p.ctx_lens[r] - q_len;
    const int key_hi = pos0 + row0 + rows_here - 1;
    const int key_lo = p.window > 0 ? max(0, pos0 + row0 - p.window + 1) : 0;
    const int t_begin = key_lo / BN, n_tiles = key_hi / BN + 1 - t_begin;
    // a key tile needs no mask if every row of the CTA sees all of it
    const int tile_pos_min = pos0 + row0;
    const int tile_lo_max = p.window > 0 ? max(0, pos0 + row0 + rows_here - 1 - p.window + 1) : 0;

    extern __shared__ __align__(1024) unsigned char smem_raw[];
    unsigned char* base = reinterpret_cast<unsigned char*>(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    unsigned char* q_s = base;                // [halves][128 rows][64]: head size 128 only
    unsigned char* kv_s = base + Sh::Q_BYTES;  // [STAGES][keys | values], each [64-wide pieces][64 keys][64]
    __shared__ __align__(8) unsigned long long q_full, k_full[STAGES], k_empty[STAGES], v_full[STAGES], v_empty[STAGES], s_full[NBUF], s_empty[NBUF], p_full, o_full;
    __shared__ unsigned tmem_base;
    __shared__ int gave_up;

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        tma::mbar_init(&q_full, Sh::Q_IN_TMEM ? 4 : 1);
#pragma unroll
        for (int s = 0; s < STAGES; ++s) {
            tma::mbar_init(&k_full[s], 1);
            tma::mbar_init(&k_empty[s], 1);
            tma::mbar_init(&v_full[s], 1);
            tma::mbar_init(&v_empty[s], 1);
        }
#pragma unroll
        for (int b = 0; b < NBUF; ++b) {
            tma::mbar_init(&s_full[b], 1);
            tma::mbar_init(&s_empty[b], 4);
        }
        tma::mbar_init(&p_full, 4);
        tma::mbar_init(&o_full, 1);
        gave_up = 0;
        tma::mbar_fence_init();
        tma::prefetch_map(&kvmap);
        if (!Sh::Q_IN_TMEM) tma::prefetch_map(&qmap);
    }
    if (warp == 5) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(tma::smem_addr(&tmem_base)), "n"(TMEM_COLS) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
    pdl_trigger();
    pdl_wait();  // the queries and the step's keys and values come from the kernels before

    auto fail = [&]() {
        gave_up = 1;
        if (tp.error_flag) atomicExch(tp.error_flag, 1);
    };

    if (warp == 4 || warp == 6) {
        // ---- producers: warp 4 brings the queries and the keys, warp 6 the values ----
        // Keys and values have rings of their own: a stage of keys is free again as soon as its scores are computed,
        // which is more than a tile before the values of the same tile have been used, so the keys of three tiles on
        // are requested that much earlier (with one ring for both, the scores waited for their keys).
        const bool is_v = warp == 6;
        unsigned long long* full = is_v ? v_full : k_full;
        unsigned long long* empty = is_v ? v_empty : k_empty;
        const int ps = p.page_size, pages_per_tile = BN / ps;
        const int lp_lo = key_lo / ps, lp_hi = key_hi / ps;
        const int* table = p.page_table + (size_t)r * p.table_width;
        if (!Sh::Q_IN_TMEM && !is_v && lane == 0) {
            tma::mbar_expect_tx(&q_full, Sh::Q_BYTES);
#pragma unroll
            for (int h = 0; h < K_HALVES; ++h) tma::load_2d(q_s + (size_t)h * (BM * 128), &qmap, q_head * KD + h * 64, q_begin + row0, &q_full);
        }
        // One box per page and 64-wide piece, each issued by a lane of its own (a thread's TMA instructions follow one another slowly;
        // several threads' overlap).  The page table is read 32 entries at a time; a page outside the needed range is
        // replaced by one inside it.
        const int first_page = t_begin * pages_per_tile, halves = is_v ? V_HALVES : K_HALVES;
        const int lane0 = is_v ? 0 : (q_head - head * tp.maps) * KD;  // where a row's lanes of this map begin
        int my_page = 0, loaded_from = -32;
        bool alive = true;
        for (int j = 0; j < n_tiles && alive; ++j) {
            const int s = j % STAGES, idx0 = j * pages_per_tile;
            if (idx0 >= loaded_from + 32) {  // pages_per_tile divides 32: a tile's pages lie in one batch
                loaded_from = idx0;
                my_page = table[min(max(first_page + idx0 + lane, lp_lo), lp_hi)];
            }
            if (lane == 0) {
                if (gave_up || (j >= STAGES && !tma::mbar_wait(&empty[s], ((j / STAGES) - 1) & 1))) {
                    if (!gave_up) fail();
                    alive = false;
                } else {
                    tma::mbar_expect_tx(&full[s], is_v ? Sh::V_BYTES : K_BYTES);
                }
            }
            alive = __shfl_sync(0xffffffffu, (int)alive, 0) != 0;
            const int in_tile = lane / halves, half = lane % halves;
            const int page = __shfl_sync(0xffffffffu, my_page, (idx0 - loaded_from + in_tile) & 31);
            if (alive && in_tile < pages_per_tile) {
                unsigned char* dst = kv_s + (size_t)s * STAGE_BYTES + (size_t)is_v * K_BYTES + (size_t)half * (BN * 128) + (size_t)in_tile * ps * 128;
                tma::load_2d(dst, &kvmap, lane0 + half * 64, ((page * 2 + (int)is_v) * p.KV + kvh) * ps, &full[s]);
            }
        }
    } else if (warp == 5) {
        // ---- issuer of the scores: S[j % 2] = Q K_j^T, as soon as the keys are there and the buffer has been read ----
        // One thread spends about a hundred cycles on every tcgen05.mma it issues and sixty on a commit, so the two
        // products of a tile have an issuing thread each: together in one thread they, not the softmax, set the pace.
        // Both products take their A operand (queries, probabilities) from tensor memory: read from shared memory, a
        // 128 x 64 x 16 step would want 6 KB in 32 cycles, more than shared memory gives.
        if (lane == 0) {
            constexpr unsigned IDESC_QK = umma::idesc_bf16(BM, BN, false);
            const unsigned q_tmem = tmem_base + Q_COL;
            bool ok = tma::mbar_wait(&q_full, 0);
            for (int j = 0; j < n_tiles && ok && !gave_up; ++j) {
                ok = tma::mbar_wait(&k_full[j % STAGES], (j / STAGES) & 1) &&
                     (j < NBUF || tma::mbar_wait(&s_empty[j % NBUF], ((j / NBUF) - 1) & 1));
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
                const unsigned char* k_tile = kv_s + (size_t)(j % STAGES) * STAGE_BYTES;
#pragma unroll
                for (int k = 0; k < KD / 16; ++k) {  // 16 of the head's lanes a step: piece k / 4 of the tile, 32 bytes further per step
                    const unsigned long long k_desc = umma::desc_sw128(k_tile + (size_t)(k / 4) * (BN * 128)) + 2 * (k % 4);
                    if constexpr (Sh::Q_IN_TMEM) {
                        umma::mma_bf16_ts(tmem_base + (j % NBUF) * BN, q_tmem + 8 * k, k_desc, IDESC_QK, k != 0);
                    } else {
                        const unsigned long long q_desc = umma::desc_sw128(q_s + (size_t)(k / 4) * (BM * 128)) + 2 * (k % 4);
                        umma::mma_bf16(tmem_base + (j % NBUF) * BN, q_desc, k_desc, IDESC_QK, k != 0);
                    }
                }
                umma::commit(&s_full[j % NBUF]);
                umma::commit(&k_empty[j % STAGES]);
            }
            if (!ok) fail();
        }
    } else if (warp == 7) {
        // ---- issuer of the second product: O += P_j V_j, as soon as the probabilities and the values are there ----
        if (lane == 0) {
            constexpr unsigned IDESC_PV = umma::idesc_bf16(BM, VD, true);
            const unsigned o_tmem = tmem_base + O_COL, p_tmem = tmem_base + P_COL;
            bool ok = true;
            for (int j = 0; j < n_tiles && ok && !gave_up; ++j) {
                const int s = j % STAGES;
                ok = tma::mbar_wait(&v_full[s], (j / STAGES) & 1) && tma::mbar_wait(&p_full, j & 1);
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
                // the values lie [key][d]: B with N contiguous; 16 keys are two atoms of 8 rows, 2048 bytes further per step
                // (a head of 128 lanes is two such pieces side by side, BN * 128 bytes apart: the leading offset)
                const unsigned long long v_desc = umma::desc_sw128(kv_s + (size_t)s * STAGE_BYTES + K_BYTES, (V_HALVES > 1 ? BN * 128 : 1024) >> 4);
#pragma unroll
                for (int k = 0; k < BN / 16; ++k)  // the output accumulates over the tiles
                    umma::mma_bf16_ts(o_tmem, p_tmem + 8 * k, v_desc + (2048 >> 4) * k, IDESC_PV, k != 0 || j != 0);
                umma::commit(&o_full);
                umma::commit(&v_empty[s]);
            }
            if (!ok) fail();
        }
    } else {
        // ---- softmax: thread = query row = lane of tensor memory ----
        const int row = warp * 32 + lane, tok = row0 + row;
        const bool row_ok = tok < q_len;
        const int pos = pos0 + tok;
        const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
        const unsigned lane_base = tmem_base + ((unsigned)(warp * 32) << 16);
        float m_run = -INFINITY, l_run = 0.f;
        bool ok = true;
        const unsigned o_taddr = lane_base + O_COL;
        if constexpr (Sh::Q_IN_TMEM) {  // the row's queries, as they lie in memory (two to a word), into the row's lane of tensor memory
            unsigned qw[32];
            const uint4* src = reinterpret_cast<const uint4*>(p.q + (size_t)(q_begin + tok) * p.q_stride + (size_t)q_head * KD);
#pragma unroll
            for (int c = 0; c < KD / 8; ++c) {
                const uint4 u = row_ok ? src[c] : make_uint4(0, 0, 0, 0);
                qw[4 * c] = u.x; qw[4 * c + 1] = u.y; qw[4 * c + 2] = u.z; qw[4 * c + 3] = u.w;
            }
            umma::tmem_st32(lane_base + Q_COL, qw);
            asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(&q_full);
        }
#ifdef ATT_PROF
        long long pc[6] = {0, 0, 0, 0, 0, 0}, c0 = clock64(), c1;
#define PH(i) { c1 = clock64(); pc[i] += c1 - c0; c0 = c1; }
#else
#define PH(i)
#endif
        for (int j = 0; j < n_tiles; ++j) {
            const int key_base = (t_begin + j) * BN;
            ok = __all_sync(0xffffffffu, !gave_up && tma::mbar_wait(&s_full[j % NBUF], (j / NBUF) & 1));
            PH(0)
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
            const bool whole = key_base + BN - 1 <= tile_pos_min && key_base >= tile_lo_max && rows_here == BM;
            // the keys of this tile that the row sees are those with index (within the tile) in [see_lo, see_hi]
            const int see_lo = row_ok ? lo - key_base : BN, see_hi = row_ok ? pos - key_base : -1;
            // the row's 64 scores in one load; once they are in registers the buffer may take the scores two tiles on
            static_assert(BN == 64, "the softmax reads a tile's scores with one 64-column load");
            float v[BN];
            umma::tmem_ld64(lane_base + (j % NBUF) * BN, v);
            asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(&s_empty[j % NBUF]);  // the buffer may take the scores of a later tile
            PH(1)
            // the row's maximum (four chains, so that the comparisons do not wait for one another; the scale is
            // positive and is applied to the maximum alone)
            float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
            if (whole) {
#pragma unroll
                for (int i = 0; i < BN; ++i) mx4[i & 3] = fmaxf(mx4[i & 3], v[i]);
            } else {
#pragma unroll
                for (int i = 0; i < BN; ++i) {
                    const bool visible = i >= see_lo && i <= see_hi;
                    v[i] = visible ? v[i] : -INFINITY;
                    mx4[i & 3] = fmaxf(mx4[i & 3], v[i]);
                }
            }
            const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * p.scale_log2;
            // The output accumulates in tensor memory, scaled by 2^-m_run.  The row keeps its old shift while the new
            // maximum is less than 2^LAZY above it (any shift gives the same quotient in the end; probabilities then
            // reach 2^LAZY at most, which bfloat16 holds with its usual relative error), so the accumulated output
            // has to be rescaled only on the few tiles where a row's maximum jumps.
            const float m_cand = fmaxf(m_run, mx);
            const bool grow = m_cand > m_run + LAZY || m_run == -INFINITY;
            const float m_new = grow ? m_cand : m_run;
            const float m_use = m_new == -INFINITY ? 0.f : m_new;
            const float alpha = attn::fast_exp2(m_run - m_use);  // 1 where the shift stays
            const bool rescale = grow && m_run != -INFINITY;  // (a row that has seen no key yet has an output of zeros)
            m_run = m_new;
            PH(2)
            // the probabilities (a masked score is -inf: its probability is exactly 0), two to a word: the second
            // product's A operand, stored into the row's lane of tensor memory once the product before has read its own
            unsigned pw[BN / 2];
            float2 sum2[2] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f)};  // four chains, two per packed add
            const float2 scale2 = make_float2(p.scale_log2, p.scale_log2), shift2 = make_float2(-m_use, -m_use);
#pragma unroll
            for (int c = 0; c < BN / 8; ++c) {
#pragma unroll
                for (int i = 0; i < 8; i += 2) {
                    const float2 x = __ffma2_rn(make_float2(v[c * 8 + i], v[c * 8 + i + 1]), scale2, shift2);
                    v[c * 8 + i] = attn::fast_exp2(x.x);
                    v[c * 8 + i + 1] = attn::fast_exp2(x.y);
                    sum2[(i >> 1) & 1] = __fadd2_rn(sum2[(i >> 1) & 1], make_float2(v[c * 8 + i], v[c * 8 + i + 1]));
                }
                pw[4 * c] = attn::pack_bf16(v[c * 8], v[c * 8 + 1]);
                pw[4 * c + 1] = attn::pack_bf16(v[c * 8 + 2], v[c * 8 + 3]);
                pw[4 * c + 2] = attn::pack_bf16(v[c * 8 + 4], v[c * 8 + 5]);
                pw[4 * c + 3] = attn::pack_bf16(v[c * 8 + 6], v[c * 8 + 7]);
            }
            l_run = l_run * alpha + ((sum2[0].x + sum2[0].y) + (sum2[1].x + sum2[1].y));
            PH(3)
            // The product of the tile before has had this tile's softmax to finish in.  Its barrier is waited for at
            // every tile, needed or not: a phase is told from the one two before it only by its parity, and a warp
            // that skipped phases could take an old one for the one it wants.
            // It has also read the probabilities of the tile before, whose place this tile's take below.
            if (j > 0) {
                ok = __all_sync(0xffffffffu, !gave_up && tma::mbar_wait(&o_full, (j - 1) & 1));
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
            }
            if (__any_sync(0xffffffffu, rescale)) {
                // this tile's product must not start before the rows are rescaled: the issuer learns of the
                // probabilities only below
                const float a = rescale ? alpha : 1.f;
                const float2 a2 = make_float2(a, a);
#pragma unroll 1
                for (int h = 0; h < V_HALVES; ++h) {
                    float o[64];
                    umma::tmem_ld64(o_taddr + 64 * h, o);
#pragma unroll
                    for (int i = 0; i < 64; i += 2) {
                        const float2 r = __fmul2_rn(make_float2(o[i], o[i + 1]), a2);
                        o[i] = r.x;
                        o[i + 1] = r.y;
                    }
                    umma::tmem_st64(o_taddr + 64 * h, o);
                }
            }
            PH(4)
            umma::tmem_st32(lane_base + P_COL, pw);
            asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(&p_full);
            PH(5)
        }
#ifdef ATT_PROF
        if (threadIdx.x == 0 && blockIdx.x == 3 && (blockIdx.y % 5) == 0)
            printf("tile %d n_tiles %d: per tile wait_s %lld ld %lld max %lld exp+store %lld o_wait %lld arrive %lld total %lld\n", tile, n_tiles,
                   pc[0] / n_tiles, pc[1] / n_tiles, pc[2] / n_tiles, pc[3] / n_tiles, pc[4] / n_tiles, pc[5] / n_tiles,
                   (pc[0] + pc[1] + pc[2] + pc[3] + pc[4] + pc[5]) / n_tiles);
#endif
        if (ok && n_tiles > 0) ok = __all_sync(0xffffffffu, !gave_up && tma::mbar_wait(&o_full, (n_tiles - 1) & 1));
        if (!ok) {
            if (lane == 0) fail();
        } else if (n_tiles > 0) {
            asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
            float inv = 1.f / l_run;
            __nv_bfloat16* dst = p.out + (size_t)(q_begin + tok) * p.out_stride + (size_t)head * VD;
            if (tp.gate && row_ok) inv /= 1.f + expf(-tp.gate[(size_t)(q_begin + tok) * tp.gate_token + head]);
            if (tp.turn) {
                const float4* cs = reinterpret_cast<const float4*>(tp.turn + (size_t)(q_begin + tok) * (VD / 2));  // two pairs each
#pragma unroll 1
                for (int h = 0; h < VD / 2; h += 32) {
                    float a[32], b[32];
                    umma::tmem_ld32(o_taddr + h, a);
                    umma::tmem_ld32(o_taddr + VD / 2 + h, b);
                    if (row_ok) {
#pragma unroll
                        for (int i = 0; i < 32; i += 2) {
                            const float4 t = cs[(h + i) >> 1];
                            const float u0 = a[i] * inv, v0 = b[i] * inv, u1 = a[i + 1] * inv, v1 = b[i + 1] * inv;
                            a[i] = u0 * t.x + v0 * t.y;
                            b[i] = v0 * t.x - u0 * t.y;
                            a[i + 1] = u1 * t.z + v1 * t.w;
                            b[i + 1] = v1 * t.z - u1 * t.w;
                        }
#pragma unroll
                        for (int c = 0; c < 4; ++c) {
                            *reinterpret_cast<uint4*>(dst + h + c * 8) =
                                make_uint4(attn::pack_bf16(a[c * 8], a[c * 8 + 1]), attn::pack_bf16(a[c * 8 + 2], a[c * 8 + 3]),
                                           attn::pack_bf16(a[c * 8 + 4], a[c * 8 + 5]), attn::pack_bf16(a[c * 8 + 6], a[c * 8 + 7]));
                            *reinterpret_cast<uint4*>(dst + VD / 2 + h + c * 8) =
                                make_uint4(attn::pack_bf16(b[c * 8], b[c * 8 + 1]), attn::pack_bf16(b[c * 8 + 2], b[c * 8 + 3]),
                                           attn::pack_bf16(b[c * 8 + 4], b[c * 8 + 5]), attn::pack_bf16(b[c * 8 + 6], b[c * 8 + 7]));
                        }
                    }
                }
            } else
#pragma unroll 1
            for (int h = 0; h < V_HALVES; ++h) {
                float o[64];
                umma::tmem_ld64(o_taddr + 64 * h, o);  // (by all lanes of the warp: the load is the warp's)
                if (row_ok && tp.raw) {
                    float* raw = tp.raw + ((size_t)(q_begin + tok) * (p.H * tp.maps) + q_head) * VD + 64 * h;
#pragma unroll
                    for (int c = 0; c < 64; c += 4)
                        *reinterpret_cast<float4*>(raw + c) = make_float4(o[c] * inv, o[c + 1] * inv, o[c + 2] * inv, o[c + 3] * inv);
                } else if (row_ok) {
#pragma unroll
                    for (int c = 0; c < 8; ++c) {
                        uint4 u;
                        u.x = attn::pack_bf16(o[c * 8] * inv, o[c * 8 + 1] * inv);
                        u.y = attn::pack_bf16(o[c * 8 + 2] * inv, o[c * 8 + 3] * inv);
                        u.z = attn::pack_bf16(o[c * 8 + 4] * inv, o[c * 8 + 5] * inv);
                        u.w = attn::pack_bf16(o[c * 8 + 6] * inv, o[c * 8 + 7] * inv);
                        *reinterpret_cast<uint4*>(dst + 64 * h + c * 8) = u;
                    }
                }
            }
        }
    }
    // after a failed wait, copies may still be on their way into this CTA's shared memory: wait for them (bounded)
    if (gave_up && threadIdx.x == 0) {
        for (int j = max(0, n_tiles - STAGES); j < n_tiles; ++j) {
            tma::mbar_wait(&k_full[j % STAGES], (j / STAGES) & 1);
            tma::mbar_wait(&v_full[j % STAGES], (j / STAGES) & 1);
        }
    }
    // everyone is done with tensor memory: the allocating warp gives it back
    asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
    __syncthreads();
    if (warp == 5) {
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem_base), "n"(TMEM_COLS) : "memory");
    }
}

// Two maps' results [tokens, H, 2, VD] (32-bit) become a head's: u = a1 - weight * a2, u / sqrt(mean(u^2) + eps) * scale, bfloat16.
// A warp a (token, head); tokens of requests with fewer than min_tokens tokens are another kernel's.
template <int VD>
__global__ void __launch_bounds__(256)
join_maps_kernel(const float* __restrict__ raw, const int* __restrict__ token_request, const int* __restrict__ cu_tokens, int min_tokens,
                 int n_tokens, int H, float weight, float eps, float scale, __nv_bfloat16* __restrict__ out, long long out_token) {
    constexpr int W = VD / 32;  // neighbouring lanes of a head a thread holds
    pdl_trigger();
    const long long item = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    if (item >= (long long)n_tokens * H) return;
    const int t = (int)(item / H), h = (int)(item - (long long)t * H), r = token_request[t];
    if (cu_tokens[r + 1] - cu_tokens[r] < min_tokens) return;
    pdl_wait();
    const float* a = raw + (size_t)item * 2 * VD + lane * W;
    float u[W], ss = 0.f;
#pragma unroll
    for (int e = 0; e < W; e += 2) {
        const float2 x = *reinterpret_cast<const float2*>(a + e), y = *reinterpret_cast<const float2*>(a + VD + e);
        u[e] = x.x - weight * y.x;
        u[e + 1] = x.y - weight * y.y;
        ss = fmaf(u[e], u[e], fmaf(u[e + 1], u[e + 1], ss));
    }
    const float norm = scale / sqrtf(warp_sum(ss) / (float)VD + eps);
    __nv_bfloat16* o = out + (long long)t * out_token + (long long)h * VD + lane * W;
#pragma unroll
    for (int e = 0; e < W; e += 2) *reinterpret_cast<__nv_bfloat162*>(o + e) = __floats2bfloat162_rn(u[e] * norm, u[e + 1] * norm);
}

}  // namespace

// The fewest tokens a request must bring for this kernel to take it (its CTAs are 128 tokens of one head).
LLM_EXPORT int llm_attention_tcgen05_min_tokens() { return 128; }

namespace {
template <int KD, int VD>
int launch_tcgen05(const TcParams& tp, const void* q, int q_stride, int n_tokens, const void* pool, long long kv_rows, int row_lanes,
                   int page_size, unsigned grid_y, cudaStream_t stream) {
    using Sh = Shape<KD, VD>;
    // one box of keys or values: a page's rows, 64 of the head's lanes; one box of queries: 128 tokens, 64 lanes of a head
    const CUtensorMap* kvmap = tma::cached_map_2d_bf16(pool, (uint64_t)kv_rows, (uint64_t)row_lanes, (uint64_t)row_lanes, (uint32_t)page_size, 64, CU_TENSOR_MAP_SWIZZLE_128B);
    const CUtensorMap* qmap = Sh::Q_IN_TMEM ? kvmap
                                            : tma::cached_map_2d_bf16(q, (uint64_t)n_tokens, (uint64_t)tp.a.H * tp.maps * KD, (uint64_t)q_stride, BM, 64, CU_TENSOR_MAP_SWIZZLE_128B);
    if (!kvmap || !qmap) return LLM_ERR_UNSUPPORTED;
    static bool configured = false;  // per head size
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(attention_tcgen05_kernel<KD, VD>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)Sh::SMEM);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    return launch_pdl(attention_tcgen05_kernel<KD, VD>, dim3((unsigned)(tp.a.H * tp.maps), grid_y), dim3(THREADS), Sh::SMEM, stream, tp, *qmap, *kvmap);
}

struct Differential {  // how two maps meet (raw == null: one map a head)
    float* raw;
    float weight, eps, scale;
    const int* token_request;
};

int attention_tcgen05(const void* q, int q_stride, void* out, int out_stride, const void* pool, long long pool_pages, const int* page_table,
                      int table_width, const int* cu_tokens, const int* ctx_lens, int requests, int n_tokens, int H, int KV, int KD, int VD,
                      int row_lanes, int page_size, int window, float scale, int min_tokens, int max_tokens, const float2* turn, const float* gate,
                      long long gate_token, const Differential& diff, int* error_flag, cudaStream_t stream) {
    if (n_tokens <= 0 || requests <= 0 || max_tokens < min_tokens) return 0;
    const bool sizes = (KD == 64 && (VD == 64 || VD == 128)) || (KD == 128 && VD == 128);
    if (!sizes || (page_size != 8 && page_size != 16 && page_size != 32 && page_size != 64)) return LLM_ERR_UNSUPPORTED;
    const int maps = diff.raw ? 2 : 1;
    if (H <= 0 || KV <= 0 || H % KV || table_width <= 0 || min_tokens < 1 || !(scale > 0.f) || row_lanes < maps * KD || row_lanes < VD ||
        (diff.raw && (turn || gate || !diff.token_request)))
        return LLM_ERR_BAD_ARGUMENT;
    if ((q_stride & 7) || (out_stride & 7) || ((uintptr_t)q & 15) || ((uintptr_t)out & 15) || ((uintptr_t)pool & 127) || q_stride < H * maps * KD ||
        (row_lanes & 7) || ((uintptr_t)turn & 15) || ((uintptr_t)diff.raw & 15))
        return LLM_ERR_UNSUPPORTED;
    const long long kv_rows = pool_pages * 2 * KV * page_size;
    if (kv_rows <= 0 || kv_rows > 0x7fffffffLL) return LLM_ERR_UNSUPPORTED;
    TcParams tp = {};
    tp.a.q = (const __nv_bfloat16*)q;
    tp.a.q_stride = q_stride;
    tp.a.out = (__nv_bfloat16*)out;
    tp.a.out_stride = out_stride;
    tp.a.page_table = page_table;
    tp.a.table_width = table_width;
    tp.a.cu_tokens = cu_tokens;
    tp.a.ctx_lens = ctx_lens;
    tp.a.H = H;
    tp.a.KV = KV;
    tp.a.G = H / KV;
    tp.a.page_size = page_size;
    tp.a.window = window;
    tp.a.scale_log2 = scale * 1.4426950408889634f;
    tp.min_tokens = min_tokens;
    tp.tiles_per_request = (max_tokens + BM - 1) / BM;
    tp.error_flag = error_flag;
    tp.maps = maps;
    tp.raw = diff.raw;
    tp.turn = turn;
    tp.gate = gate;
    tp.gate_token = gate_token;
    const long long y = (long long)requests * tp.tiles_per_request;
    if (y > 65535) return LLM_ERR_UNSUPPORTED;
    int code;
    if (KD == 64 && VD == 64) code = launch_tcgen05<64, 64>(tp, q, q_stride, n_tokens, pool, kv_rows, row_lanes, page_size, (unsigned)y, stream);
    else if (KD == 64) code = launch_tcgen05<64, 128>(tp, q, q_stride, n_tokens, pool, kv_rows, row_lanes, page_size, (unsigned)y, stream);
    else code = launch_tcgen05<128, 128>(tp, q, q_stride, n_tokens, pool, kv_rows, row_lanes, page_size, (unsigned)y, stream);
    if (code != 0 || maps == 1) return code;
    const long long items = (long long)n_tokens * H;
    auto join = [&](auto kernel) {
        return launch_pdl(kernel, dim3((unsigned)((items + 7) / 8)), dim3(256), 0, stream, (const float*)diff.raw, diff.token_request, cu_tokens, min_tokens,
                          n_tokens, H, diff.weight, diff.eps, diff.scale, (__nv_bfloat16*)out, (long long)out_stride);
    };
    return VD == 64 ? join(join_maps_kernel<64>) : join(join_maps_kernel<128>);
}
}  // namespace

// Attention of the requests that bring at least min_tokens tokens (others are left untouched: another kernel's).
// q: bfloat16 rows of q_stride elements that start with the H query heads; out: [tokens, H * D] with row stride
// out_stride; pool: one layer's plane [pool_pages, 2, KV, page_size, D]; max_tokens: the most tokens of any request.
// Takes head sizes 64 and 128, pages of 8, 16, 32 or 64 keys, 16-byte aligned rows; else LLM_ERR_UNSUPPORTED (nothing ran).
LLM_EXPORT int llm_attention_tcgen05(const void* q, int q_stride, void* out, int out_stride, const void* pool, long long pool_pages,
                                     const int* page_table, int table_width, const int* cu_tokens, const int* ctx_lens,
                                     int requests, int n_tokens, int H, int KV, int D, int page_size, int window, float scale,
                                     int min_tokens, int max_tokens, int* error_flag, cudaStream_t stream) {
    return attention_tcgen05(q, q_stride, out, out_stride, pool, pool_pages, page_table, table_width, cu_tokens, ctx_lens, requests, n_tokens, H, KV, D, D,
                             D, page_size, window, scale, min_tokens, max_tokens, nullptr, nullptr, 0, Differential{}, error_flag, stream);
}

// The same with keys of KD and values of VD lanes (64 and 64, 64 and 128, 128 and 128) in rows of row_lanes; `turn` [tokens, VD / 2] pairs
// (cos, sin) or null: values that turn back; `gate` (row pitch gate_token) or null: one gate a head; `raw` [tokens, H, 2, VD] (32-bit
// scratch) or null: two score maps a head, whose results meet as u / sqrt(mean(u^2) + diff_eps) * diff_scale, u = a1 - diff_weight * a2
// (a second launch; without turn and gate).
LLM_EXPORT int llm_attention_tcgen05_general(const void* q, int q_stride, void* out, int out_stride, const void* pool, long long pool_pages,
                                             const int* page_table, int table_width, const int* token_request, const int* cu_tokens,
                                             const int* ctx_lens, int requests, int n_tokens, int H, int KV, int KD, int VD, int row_lanes,
                                             int page_size, int window, float scale, int min_tokens, int max_tokens, const void* turn,
                                             const float* gate, long long gate_token, float* raw, float diff_weight, float diff_eps,
                                             float diff_scale, int* error_flag, cudaStream_t stream) {
    const Differential diff = {raw, diff_weight, diff_eps, diff_scale, token_request};
    return attention_tcgen05(q, q_stride, out, out_stride, pool, pool_pages, page_table, table_width, cu_tokens, ctx_lens, requests, n_tokens, H, KV, KD, VD,
                             row_lanes, page_size, window, scale, min_tokens, max_tokens, (const float2*)turn, gate, gate_token, diff, error_flag, stream);
}
