// Latent attention: what the decode GEMVs do for it (epilogues and prologues; the attention kernels themselves are in
// latent_attention.cuh).
//
// A token leaves one row behind, shared by all heads: its RMS-normed latent c [rank] and one rotated key part
// [rot].  A head's key is (W_uk c, rotated part) and its value W_uv c.  Both expansions are linear in c, so they are
// applied on the other side: the score is  q_plain . (W_uk c) = (W_uk^T q_plain) . c  and the weighted sum of the values is
// W_uv (sum_j p_j c_j).  Per head the query becomes a row (W_uk^T q_plain, q_rot) of the cache row's width, attention is a
// dot product with cache rows and a weighted sum of their latent parts, and nothing of the size heads x keys x dim is
// ever formed.  One decode step of a layer:
//
//   1. input GEMV   rows  plain queries | rotated queries | latent | rotated key part | gates  (all read the same
//                   normed input): plain queries and raw latent to FP32 buffers, rotated parts turned and stored where
//                   they belong, gates through the sigmoid
//   2. query GEMV   per head: W_uk^T q_plain into the head's query row; one more CTA norms the latent into the cache row
//   3. attention    splits over the keys of the window, partial results with their maximum and sum
//   4. value GEMV   per head: puts the splits together, W_uv times the result, times the head's gate
//   5. output GEMV  with the residual, like every other mixer
//
// Widths inside the engine: rank_pitch and rot part are rounded up to 16 elements in query and cache rows (row_width in
// all), inputs per head to 64 elements; the padding is zero in the weights and in the cache.
#pragma once
#include "common.cuh"

namespace lpp {

constexpr int kLatentMaxSplits = 32;   // key ranges of one attention launch
constexpr int kLatentPartTail = 4;     // floats behind a partial result: maximum, sum, padding to 16 bytes

struct LatentArgs {
    int heads, dim, rot, vdim, rank;            // true sizes (per head: dim plain, rot rotated, vdim value)
    int dim_pitch;                              // plain query inputs of one head in q_plain
    int rank_pitch, row_width;                  // latent part and whole of a query / cache row
    int vdim_rows;                              // rows of one head in the value matrix (vdim rounded up to even)
    int q_plain_rows, q_rot_rows, latent_rows;  // sections of the input matrix, each an even number of rows
    int cache_f32;                              // query and cache rows are FP32 instead of FP16
    const float2* rope;                         // [positions][rot / 2] (cos, sin), magnitude included
    float* q_plain;                             // [heads][dim_pitch]
    float* latent;                              // [latent_rows], not normed
    float* gate;                                // [heads]
    void* query;                                // [heads][row_width]
    void* cache;                                // [positions][row_width]
    const float* norm_w;                        // latent norm weight [rank]
    float norm_eps;
    const float* part;                          // [heads][max_splits][rank_pitch + kLatentPartTail]
    int window, max_splits, min_chunk;
};

// The keys that queries at positions lo .. hi can see between them, and how they are cut into splits.  Evaluated alike
// by the attention kernel and by whoever puts its partial results together.
struct LatentSpan {
    int first, n_keys, chunk, n_eff;
};
__host__ __device__ inline LatentSpan latent_span(int lo, int hi, int window, int max_splits, int min_chunk) {
    LatentSpan s;
    s.first = (window > 0 && lo - window + 1 > 0) ? lo - window + 1 : 0;
    s.n_keys = hi - s.first + 1;
    s.chunk = (s.n_keys + max_splits - 1) / max_splits;
    s.chunk = (s.chunk + 15) / 16 * 16;
    if (s.chunk < min_chunk) s.chunk = min_chunk;
    s.n_eff = (s.n_keys + s.chunk - 1) / s.chunk;
    return s;
}

__device__ __forceinline__ void latent_put(void* base, int f32, size_t i, float v) {
    if (f32)
        reinterpret_cast<float*>(base)[i] = v;
    else
        reinterpret_cast<__half*>(base)[i] = __float2half_rn(v);
}

// Epilogue of the input GEMV: rows row and row + 1 (row even).
__device__ __forceinline__ void latent_in_rows(const LatentArgs& L, StepState* st, int seq_len, int row, float v0, float v1) {
    const int pos = st->pos;
    if (pos < 0 || pos >= seq_len) {
        atomicOr(&st->status, kStatusBadPos);
        return;
    }
    int r = row;
    if (r < L.q_plain_rows) {
        if (r < L.heads * L.dim) L.q_plain[(size_t)(r / L.dim) * L.dim_pitch + r % L.dim] = v0;
        ++r;
        if (r < L.heads * L.dim) L.q_plain[(size_t)(r / L.dim) * L.dim_pitch + r % L.dim] = v1;
        return;
    }
    r -= L.q_plain_rows;
    const bool is_q = r < L.q_rot_rows;
    if (!is_q) {
        r -= L.q_rot_rows;
        if (r < L.latent_rows) {
            *reinterpret_cast<float2*>(L.latent + r) = make_float2(v0, v1);
            return;
        }
        r -= L.latent_rows;
        if (r >= L.rot) {
            r -= L.rot;
            if (r < L.heads) L.gate[r] = sigmoid_f(v0);
            if (r + 1 < L.heads) L.gate[r + 1] = sigmoid_f(v1);
            return;
        }
    }
    // a rotated pair, of a head's query or of the shared key part
    const int h = is_q ? r / L.rot : 0, j = r - h * L.rot;
    const float2 cs = __ldg(L.rope + (size_t)pos * (L.rot >> 1) + (j >> 1));
    const float r0 = __fsub_rn(__fmul_rn(v0, cs.x), __fmul_rn(v1, cs.y));
    const float r1 = __fadd_rn(__fmul_rn(v1, cs.x), __fmul_rn(v0, cs.y));
    const size_t at = (size_t)(is_q ? h : pos) * L.row_width + L.rank_pitch + j;
    void* base = is_q ? L.query : L.cache;
    latent_put(base, L.cache_f32, at, r0);
    latent_put(base, L.cache_f32, at + 1, r1);
}

// Epilogue of the query GEMV: rank_pitch rows per head (the ones beyond rank have zero weights).
__device__ __forceinline__ void latent_query_rows(const LatentArgs& L, int row, float v0, float v1) {
    const int h = row / L.rank_pitch, r = row - h * L.rank_pitch;
    const size_t at = (size_t)h * L.row_width + r;
    latent_put(L.query, L.cache_f32, at, v0);
    latent_put(L.query, L.cache_f32, at + 1, v1);
}

// Epilogue of the value GEMV: vdim_rows rows per head; out is the output projection's input, heads one after the other.
__device__ __forceinline__ void latent_value_rows(const LatentArgs& L, float* out, int row, float v0, float v1) {
    const int h = row / L.vdim_rows, r = row - h * L.vdim_rows;
    const float g = __ldcg(L.gate + h);
    float* o = out + (size_t)h * L.vdim + r;
    if (r < L.vdim) o[0] = v0 * g;
    if (r + 1 < L.vdim) o[1] = v1 * g;
}

// The raw latent of this token -> RMS norm -> its cache row.  NT threads; scratch holds NT / 32 floats and is free again
// when the call returns.
template <int NT>
__device__ __forceinline__ void latent_norm_to_cache(const LatentArgs& L, const StepState* st, int seq_len, float* scratch, int tid) {
    const int pos = st->pos;
    const bool ok = pos >= 0 && pos < seq_len;
    float ss = 0.f;
    for (int i = tid; i < L.rank; i += NT) {
        const float v = __ldcg(L.latent + i);
        ss = fmaf(v, v, ss);
    }
    ss = warp_sum(ss);
    if ((tid & 31) == 0) scratch[tid >> 5] = ss;
    consumer_barrier(NT);
    float tot = 0.f;
#pragma unroll
    for (int w = 0; w < NT / 32; ++w) tot += scratch[w];
    const float scale = __fdiv_rn(1.0f, __fsqrt_rn(__fadd_rn(__fdiv_rn(tot, (float)L.rank), L.norm_eps)));
    if (ok)
        for (int i = tid; i < L.rank; i += NT)
            latent_put(L.cache, L.cache_f32, (size_t)pos * L.row_width + i,
                       __fmul_rn(__fmul_rn(__ldcg(L.latent + i), scale), __ldg(L.norm_w + i)));
    consumer_barrier(NT);
}

// Weights of the attention splits of heads first .. first + n - 1: wt[g][s] = exp(m_s - max m) / sum of l.  Returns the
// number of splits in use.  One warp per head, a lane per split.
template <int NT>
__device__ __forceinline__ int latent_split_weights(const LatentArgs& L, const StepState* st, int seq_len, float* wt, int tid,
                                                    int first, int n) {
    const int pos = st->pos;
    if (pos < 0 || pos >= seq_len) return 0;
    const int n_eff = latent_span(pos, pos, L.window, L.max_splits, L.min_chunk).n_eff;
    const int lane = tid & 31, ps = L.rank_pitch + kLatentPartTail;
    for (int g = tid >> 5; g < n; g += NT / 32) {
        const float* p = L.part + ((size_t)(first + g) * L.max_splits + lane) * ps + L.rank_pitch;
        const float m = lane < n_eff ? __ldcg(p) : -INFINITY, l = lane < n_eff ? __ldcg(p + 1) : 0.f;
        const float mm = warp_max(m);
        const float e = lane < n_eff ? expf(m - mm) : 0.f;
        const float sum = warp_sum(e * l);
        wt[g * kLatentMaxSplits + lane] = __fdiv_rn(e, sum);
    }
    return n_eff;
}
// Elements k .. k + 3 of head h's attended latent.
__device__ __forceinline__ float4 latent_combine4(const LatentArgs& L, const float* wt, int h, int n_eff, int k) {
    float4 r = make_float4(0.f, 0.f, 0.f, 0.f);
    if (k >= L.rank_pitch) return r;
    const int ps = L.rank_pitch + kLatentPartTail;
    const float* p = L.part + (size_t)h * L.max_splits * ps + k;
    for (int s0 = 0; s0 < n_eff; s0 += 8) {
        float4 v[8];
#pragma unroll
        for (int i = 0; i < 8; ++i)
            if (s0 + i < n_eff) v[i] = __ldcg(reinterpret_cast<const float4*>(p + (size_t)(s0 + i) * ps));
#pragma unroll
        for (int i = 0; i < 8; ++i)
            if (s0 + i < n_eff) {
                const float w = wt[s0 + i];
                r.x = fmaf(w, v[i].x, r.x); r.y = fmaf(w, v[i].y, r.y); r.z = fmaf(w, v[i].z, r.z); r.w = fmaf(w, v[i].w, r.w);
            }
    }
    return r;
}

}  // namespace lpp
