// The arguments of attention in its general form, shared by the kernels that take it.
#pragma once

#include "common.cuh"

// Where queries, keys and values lie.  A query is one or two runs of lanes (the second may be absent): run 0 holds
// lanes [0, d0), run 1 lanes [d0, d0 + d1); each run is addressed by a token stride and a head stride.  Keys and
// values are addressed by page, key/value head and place in the page; values may be the first dv lanes of the keys
// (the same pointer and strides).
template <typename T>
struct RowsArgs {
    const T *q0, *q1;
    long long q0_token, q0_head, q1_token, q1_head;
    int d0, d1;
    T* out;
    long long out_token, out_head;
    const T *keys, *values;
    long long k_page, k_head, k_token, v_page, v_head, v_token;
    int dv;
    const int *page_table, *token_request, *cu_tokens, *ctx_lens;
    const float* slopes;  // per query head: the score of key j for the query at position i loses slope * (i - j); null: none
    int table_width, n_tokens, H, KV, page_size, window;
    int skip_from;  // > 0: requests that bring at least so many tokens are another kernel's
    // With a window, keys at positions below keep_first stay visible to every later query (0: none).  chunk > 0: a query
    // sees only keys of its own block of `chunk` positions, counted from position 0.
    int keep_first, chunk;
    float scale;
    // > 0: a score s (scaled) becomes softcap * tanh(s / softcap) before the distance bias is taken off
    float softcap;
    // Which keys: 0 all that a row sees; 1 only those cached before this step (positions before the request's first new
    // token); 2 only the step's own tokens, whose keys and values then lie token by token, not in pages: token i of the
    // flat batch at keys + i * k_token + head * k_head (lanes [0, fresh_d0)) and at keys1 + i * k1_token (the lanes
    // behind them, shared by all heads; null: all lanes at keys), its value at values + i * v_token + head * v_head.
    int key_part;
    const T* keys1;
    long long k1_token;
    int fresh_d0;
    // [n_tokens, H, 2] (or null): the row's maximum score (times log2 e) and the sum of its exponentials, for a merge of two parts; a
    // row that saw no key says (-inf, 0) and its output is not to be read
    float* stats;
    // per query head (or null): one more term exp(sinks[h]) in the softmax's denominator, with no key and no value; it is
    // not scaled and counts once
    const float* sinks;
    // [n_tokens, gate_token] float32 (or null): the output of head h, lane d is multiplied by sigmoid(gate[t, h * dv + d]),
    // or, with gate_per_head, by sigmoid(gate[t, h])
    const float* gate;
    long long gate_token;
    int gate_per_head;
    // Two score maps a head over the same values (maps = 2; 1: an ordinary head).  A head's query of map m starts m * q_map
    // elements behind its first lane, a key head's key of map m starts m * k_map behind its own, d0 lanes each (d1 = 0).
    // Every map has a softmax of its own; with a1 and a2 their outputs the head's output is u / sqrt(mean(u^2) + diff_eps)
    // * diff_scale over the head's dv lanes, u = a1 - diff_weight * a2.
    int maps;
    long long q_map, k_map;
    float diff_weight, diff_eps, diff_scale;
    // [n_tokens, dv / 2] (cos, sin) (or null): the values in the pages were turned by their own positions' angles; pair m of a
    // head's output, lanes m and m + dv/2 (turn_neighbours: 2m and 2m + 1), is turned back by the query token's row
    const float2* turn;
    int turn_neighbours;
};

// The end of one head's output: y [dv] in shared memory, complete and visible to this warp; turned back where the values were
// turned (`turn`: the token's row or null), gated (`gate`: the head's first gate or null, `gate_step` apart) and written.
template <typename T>
__device__ __forceinline__ void write_head(const float* y, int dv, int lane, const float2* turn, int neighbours, const float* gate,
                                           int gate_step, T* out) {
    auto put = [&](int d, float v) {
        if (gate) v *= 1.f / (1.f + expf(-gate[(size_t)d * gate_step]));
        out[d] = from_float<T>(v);
    };
    if (turn) {
        const int half = dv >> 1;
        for (int m = lane; m < half; m += 32) {
            const int a = neighbours ? 2 * m : m, b = neighbours ? 2 * m + 1 : m + half;
            const float2 cs = turn[m];
            const float u = y[a], v = y[b];
            put(a, u * cs.x + v * cs.y);
            put(b, v * cs.x - u * cs.y);
        }
    } else {
        for (int d = lane; d < dv; d += 32) put(d, y[d]);
    }
}

