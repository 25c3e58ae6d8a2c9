// Grouped-query attention whose values are its keys before rotation, with an optional gate on every element of the result:
// the input projection's rows and their way into query and cache rows.
//
// One projection gives a key/value head's value v and, with its first rot dimensions turned by the position, its key.  A
// position therefore leaves one row per key/value head:  v [dim], padded to 16 | turned part [rot], padded to 16.  A
// head's query row is laid out alike, with zeros where the turned dimensions' unturned values are:  0 [rot], rest of q |
// turned part of q.  The dot product of the two rows is the score and the first dim columns are the value, which is the
// shared-row attention of latent_attention.cuh (a position's traffic is dim + rot elements per key/value head instead of
// 2 dim).  One decode step of a layer:
//
//   1. input GEMV   rows  queries | keys | gates  (all read the same normed input), heads padded to an even number of
//                   rows: biases, rotation, query and cache rows, gates through the sigmoid
//   2. attention    splits over the keys of the window; the last CTA of a row tile puts them together and applies the gate
//   3. output GEMV  with bias and residual
#pragma once
#include "latent.cuh"

namespace lpp {

struct SharedKvArgs {
    int heads, kv_heads, dim, rot;  // rot: even, <= dim
    int head_rows;                  // rows of a head in the input matrix (dim rounded up to even)
    int q_rows, k_rows;             // sections of the input matrix: queries, keys, then gates (as many as queries) if any
    int rank_pitch, row_width;      // value part and whole of a query / cache row
    int cache_f32;                  // rows are FP32 instead of FP16
    int early;                      // constants may be read before the dependency wait (and so may the position)
    const float* bias;              // [q_rows + k_rows]
    const float2* rope;             // [positions][rot / 2] (cos, sin), magnitude included
    void* query;                    // [heads][row_width]
    void* cache;                    // [kv_heads][seq_len][row_width]
    float* gate;                    // [heads * dim]
};

// Row `row`: its own and its pair partner's bias, and the pair's rotation (1, 0 where nothing turns).
__device__ __forceinline__ RowPrep shared_kv_prep(const SharedKvArgs& s, int pos, int row) {
    RowPrep p;
    p.z = 1.f;
    if (row < s.q_rows + s.k_rows) {
        p.x = __ldg(s.bias + row);
        p.y = __ldg(s.bias + (row ^ 1));
        const int j = row % s.head_rows;
        if (j < s.rot) {
            const float2 cs = __ldg(s.rope + (size_t)pos * (s.rot >> 1) + (j >> 1));
            p.z = cs.x;
            p.w = cs.y;
        }
    }
    return p;
}
// v: the product of row `row`, other: that of its pair partner row ^ 1.  query / gate: this token's; pos: its position.
__device__ __forceinline__ void shared_kv_row(const SharedKvArgs& s, void* query, float* gate, int seq_len, int pos, int row, float v,
                                              float other, const RowPrep& p) {
    const bool is_q = row < s.q_rows, is_k = !is_q && row < s.q_rows + s.k_rows;
    const int r = is_q ? row : is_k ? row - s.q_rows : row - s.q_rows - s.k_rows;
    const int h = r / s.head_rows, j = r - h * s.head_rows;
    if (j >= s.dim) return;  // padding of an odd head
    if (!is_q && !is_k) {
        gate[(size_t)h * s.dim + j] = sigmoid_f(v);
        return;
    }
    v += p.x;
    other += p.y;
    void* base = is_q ? query : s.cache;
    const size_t at = (is_q ? (size_t)h : (size_t)h * seq_len + pos) * s.row_width;
    const bool turns = j < s.rot;
    latent_put(base, s.cache_f32, at + j, is_q && turns ? 0.f : v);
    if (turns) {
        const float t = (row & 1) ? __fadd_rn(__fmul_rn(v, p.z), __fmul_rn(other, p.w)) : __fsub_rn(__fmul_rn(v, p.z), __fmul_rn(other, p.w));
        latent_put(base, s.cache_f32, at + s.rank_pitch + j, t);
    }
}

}  // namespace lpp
