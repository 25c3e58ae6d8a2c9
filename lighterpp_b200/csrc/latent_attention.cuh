// Attention kernels of latent attention (latent.cuh has the scheme) and the two small kernels around them on the batched
// prompt path.
//
// In the latent space all heads share one key / value row per position, so the query rows of an attention launch are the
// (token, head) pairs, row = token * heads + head: one row block for a decode step, n_tokens x heads rows for a prompt
// block.  A CTA takes a tile of query rows and one of the splits of the keys that the tile's tokens can see (sliding
// window; a tile's tokens are neighbours, so their windows nearly coincide) and writes the unnormalised weighted sum,
// its maximum and its sum.  Whoever consumes the result puts the splits together (value GEMV when decoding,
// prefill_latent_combine_kernel in a prompt block).
#pragma once
#include "latent.cuh"
#include "prefill.cuh"

namespace lpp {

struct LatentAttnArgs {
    const void* q;      // [rows][row_width]
    const void* cache;  // [positions][row_width], this layer's
    float* part;        // [rows][max_splits][rank_pitch + kLatentPartTail]
    const StepState* st;
    int start_pos;      // position of token 0; < 0 = the step's device-resident position
    int n_tokens, heads;
    int rank_pitch, row_width;
    int window, max_splits, min_chunk;
    int seq_len;
    float scale;
};

constexpr int kLatentTile = 64;        // keys per shared-memory tile
constexpr int kLatentThreads = 256;

// ---- any sizes, FP32 or FP16 rows, FP32 arithmetic.  grid: (splits, heads, tokens)
constexpr int kLatentMaxPerThread = 8;  // latent elements of one thread: ranks up to 2048
template <typename KT>
static __global__ void __launch_bounds__(kLatentThreads) latent_attn_kernel(const LatentAttnArgs a) {
    extern __shared__ float lat_smem[];  // query row, then scores of a tile
    __shared__ float s_f, s_m, s_l;
    float* qs = lat_smem;
    float* sc = lat_smem + a.row_width;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    pdl_launch_dependents();
    pdl_wait();
    const int base = a.start_pos >= 0 ? a.start_pos : a.st->pos;
    const int pos = base + (int)blockIdx.z;
    if (base < 0 || pos >= a.seq_len) return;
    const LatentSpan sp = latent_span(pos, pos, a.window, a.max_splits, a.min_chunk);
    const int split = blockIdx.x;
    if (split >= sp.n_eff) return;
    const int k_begin = sp.first + split * sp.chunk, k_end = min(k_begin + sp.chunk, pos + 1);
    const size_t row = (size_t)blockIdx.z * a.heads + blockIdx.y;
    const KT* q = reinterpret_cast<const KT*>(a.q) + row * a.row_width;
    const KT* kc = reinterpret_cast<const KT*>(a.cache);
    for (int i = tid; i < a.row_width; i += kLatentThreads) qs[i] = to_float(q[i]);
    if (tid == 0) s_m = -INFINITY, s_l = 0.f;
    float o[kLatentMaxPerThread];
#pragma unroll
    for (int i = 0; i < kLatentMaxPerThread; ++i) o[i] = 0.f;
    __syncthreads();
    for (int k0 = k_begin; k0 < k_end; k0 += kLatentTile) {
        const int cnt = min(kLatentTile, k_end - k0);
        for (int k = warp; k < cnt; k += kLatentThreads / 32) {
            const KT* kr = kc + (size_t)(k0 + k) * a.row_width;
            float s = 0.f;
            for (int i = lane; i < a.row_width; i += 32) s = fmaf(qs[i], to_float(kr[i]), s);
            s = warp_sum(s);
            if (lane == 0) sc[k] = s * a.scale;
        }
        __syncthreads();
        if (warp == 0) {
            const float x0 = lane < cnt ? sc[lane] : -INFINITY, x1 = lane + 32 < cnt ? sc[lane + 32] : -INFINITY;
            const float m = fmaxf(s_m, warp_max(fmaxf(x0, x1)));
            const float p0 = expf(x0 - m), p1 = expf(x1 - m);  // exp(-inf) = 0
            const float l = warp_sum(p0 + p1);
            sc[lane] = p0;
            sc[lane + 32] = p1;
            if (lane == 0) {
                s_f = expf(s_m - m);
                s_l = s_l * s_f + l;
                s_m = m;
            }
        }
        __syncthreads();
        const float f = s_f;
#pragma unroll
        for (int j = 0; j < kLatentMaxPerThread; ++j) {
            const int i = tid + j * kLatentThreads;
            if (i < a.rank_pitch) {
                float acc = o[j] * f;
                const KT* kr = kc + (size_t)k0 * a.row_width + i;
#pragma unroll 8
                for (int k = 0; k < cnt; ++k) acc = fmaf(sc[k], to_float(kr[(size_t)k * a.row_width]), acc);
                o[j] = acc;
            }
        }
        __syncthreads();
    }
    float* p = a.part + (row * a.max_splits + split) * (a.rank_pitch + kLatentPartTail);
#pragma unroll
    for (int j = 0; j < kLatentMaxPerThread; ++j)
        if (tid + j * kLatentThreads < a.rank_pitch) p[tid + j * kLatentThreads] = o[j];
    if (tid == 0) {
        p[a.rank_pitch] = s_m;
        p[a.rank_pitch + 1] = s_l;
    }
}

// ---- tensor cores, FP16 rows.  grid: (splits, row tiles of 16 MT).
//
// Eight warps, MT along the query rows times WN = 8 / MT along the other direction of each product.  Query tile and
// 64-key tiles (double buffered, 16-byte asynchronous copies) lie in shared memory in rows padded by 16 bytes.  Per tile:
// scores by mma.sync m16n8k16 over the row width into shared memory (FP32); mask, running maximum, exponentials and sum
// in FP32, a few rows per warp; probabilities (FP16) times the latent part of the same tile, a warp holding 16 rows x
// NT * 8 columns of the result.
template <int MT, int NT>
static __global__ void __launch_bounds__(kLatentThreads) latent_attn_mma_kernel(const LatentAttnArgs a) {
    constexpr int kRows = 16 * MT, WN = 8 / MT, kTilesW = 8 / WN;  // kTilesW: 8-key tiles of the scores per warp
    constexpr int kScPitch = kLatentTile + 4, kPPitch = kLatentTile + 8;
    static_assert(NT % 2 == 0, "column tiles go in pairs");
    extern __shared__ __align__(128) unsigned char lm_smem[];
    const int pitch = a.row_width * 2 + 16;
    unsigned char* qs = lm_smem;
    unsigned char* kt = qs + kRows * pitch;
    float* sc = reinterpret_cast<float*>(kt + 2 * kLatentTile * pitch);
    __half* ps = reinterpret_cast<__half*>(sc + kRows * kScPitch);
    float* s_m = reinterpret_cast<float*>(ps + kRows * kPPitch);
    float* s_l = s_m + kRows;
    float* s_f = s_l + kRows;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    pdl_launch_dependents();
    // the position was written by the previous step's sampler (or comes with the launch)
    const int base = a.start_pos >= 0 ? a.start_pos : a.st->pos;
    const int n_rows = a.n_tokens * a.heads;
    const int r0 = blockIdx.y * kRows;
    const int t_lo = r0 / a.heads, t_hi = (min(r0 + kRows, n_rows) - 1) / a.heads;
    LatentSpan sp = {0, 0, 1, 0};
    if (base >= 0 && base + a.n_tokens <= a.seq_len)
        sp = latent_span(base + t_lo, base + t_hi, a.window, a.max_splits, a.min_chunk);
    const int split = blockIdx.x;
    if (split >= sp.n_eff || r0 >= n_rows) {
        pdl_wait();
        return;
    }
    const int k_begin = sp.first + split * sp.chunk, k_end = min(k_begin + sp.chunk, base + t_hi + 1);
    const int n_tiles = (k_end - k_begin + kLatentTile - 1) / kLatentTile;
    const unsigned char* cache = reinterpret_cast<const unsigned char*>(a.cache);
    const size_t row_bytes = (size_t)a.row_width * 2;
    const int pieces = a.row_width / 8;

    // rows of the tile in [lo, hi); rows at or beyond k_end are filled with zeros when `fill` is set
    auto load_keys = [&](int tile, int lo, int hi, bool fill) {
        unsigned char* dst = kt + (size_t)(tile & 1) * kLatentTile * pitch;
        const int p0 = k_begin + tile * kLatentTile;
        for (int c = tid; c < kLatentTile * pieces; c += kLatentThreads) {
            const int r = c / pieces, col = c - r * pieces, p = p0 + r;
            const bool in = p >= lo && p < hi, out = p >= k_end;
            if (in || (out && fill))
                cp_async_16(dst + (size_t)r * pitch + col * 16, in ? cache + (size_t)p * row_bytes + col * 16 : cache, in);
        }
    };
    // cache rows of earlier steps and blocks do not depend on the preceding kernels
    load_keys(0, k_begin, min(k_end, base), false);
    pdl_wait();
    load_keys(0, max(k_begin, base), k_end, true);
    for (int c = tid; c < kRows * pieces; c += kLatentThreads) {
        const int r = c / pieces, col = c - r * pieces;
        const bool in = r0 + r < n_rows;
        cp_async_16(qs + (size_t)r * pitch + col * 16,
                    reinterpret_cast<const unsigned char*>(a.q) + (in ? (size_t)(r0 + r) * row_bytes + col * 16 : 0), in);
    }
    cp_async_commit();
    if (tid < kRows) {
        s_m[tid] = -INFINITY;
        s_l[tid] = 0.f;
    }

    const int mw = warp / WN, nw = warp % WN;
    const int g = lane >> 2, tq = lane & 3, mi = lane >> 3, mr = lane & 7;
    float o[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    const uint32_t q_addr = smem_u32(qs) + (uint32_t)((mw * 16 + (mi & 1) * 8 + mr) * pitch + (mi >> 1) * 16);
    const int k_steps = a.row_width / 16;

    for (int tile = 0; tile < n_tiles; ++tile) {
        if (tile + 1 < n_tiles) {
            load_keys(tile + 1, k_begin, k_end, true);
            cp_async_commit();
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        const uint32_t ks = smem_u32(kt) + (uint32_t)((tile & 1) * kLatentTile * pitch);
        {  // scores: 16 rows x kTilesW * 8 keys per warp, two accumulators per key tile (even and odd k-steps)
            float c[kTilesW][2][4];
#pragma unroll
            for (int j = 0; j < kTilesW; ++j)
#pragma unroll
                for (int e = 0; e < 2; ++e) c[j][e][0] = c[j][e][1] = c[j][e][2] = c[j][e][3] = 0.f;
            auto step = [&](int kk, int e) {
                uint32_t qa[4];
                ldmatrix_x4(q_addr + (uint32_t)kk * 32u, qa[0], qa[1], qa[2], qa[3]);
                if constexpr (kTilesW == 1) {
                    uint32_t b0, b1;
                    ldmatrix_x2(ks + (uint32_t)((nw * 8 + mr) * pitch + kk * 32 + (mi & 1) * 16), b0, b1);
                    mma_f16_16816(c[0][e], qa[0], qa[1], qa[2], qa[3], b0, b1);
                } else {
#pragma unroll
                    for (int j = 0; j < kTilesW; j += 2) {
                        uint32_t b[4];
                        ldmatrix_x4(ks + (uint32_t)(((nw * kTilesW + j) * 8 + (mi >> 1) * 8 + mr) * pitch + kk * 32 + (mi & 1) * 16),
                                    b[0], b[1], b[2], b[3]);
                        mma_f16_16816(c[j][e], qa[0], qa[1], qa[2], qa[3], b[0], b[1]);
                        mma_f16_16816(c[j + 1][e], qa[0], qa[1], qa[2], qa[3], b[2], b[3]);
                    }
                }
            };
            int kk = 0;
#pragma unroll 4
            for (; kk + 1 < k_steps; kk += 2) {
                step(kk, 0);
                step(kk + 1, 1);
            }
            if (kk < k_steps) step(kk, 0);
#pragma unroll
            for (int j = 0; j < kTilesW; ++j) {
                float* s = sc + (mw * 16 + g) * kScPitch + (nw * kTilesW + j) * 8 + 2 * tq;
                *reinterpret_cast<float2*>(s) = make_float2(c[j][0][0] + c[j][1][0], c[j][0][1] + c[j][1][1]);
                *reinterpret_cast<float2*>(s + 8 * kScPitch) = make_float2(c[j][0][2] + c[j][1][2], c[j][0][3] + c[j][1][3]);
            }
        }
        __syncthreads();
        // mask and online softmax: 2 MT rows per warp, two keys per lane
        const int p = k_begin + tile * kLatentTile + lane;
#pragma unroll
        for (int i = 0; i < 2 * MT; ++i) {
            const int r = warp * 2 * MT + i;
            const int row = min(r0 + r, n_rows - 1);
            const int last = base + row / a.heads, lo = a.window > 0 ? last - a.window + 1 : 0;
            const float x0 = (p >= lo && p <= last && p < k_end) ? sc[r * kScPitch + lane] * a.scale : -INFINITY;
            const float x1 = (p + 32 >= lo && p + 32 <= last && p + 32 < k_end) ? sc[r * kScPitch + lane + 32] * a.scale : -INFINITY;
            const float m_old = s_m[r], m = fmaxf(m_old, warp_max(fmaxf(x0, x1)));
            const float u = m == -INFINITY ? 0.f : m;  // nothing visible to this row yet
            const float p0 = __expf(x0 - u), p1 = __expf(x1 - u);
            const float l = warp_sum(p0 + p1);
            ps[r * kPPitch + lane] = __float2half_rn(p0);
            ps[r * kPPitch + lane + 32] = __float2half_rn(p1);
            __syncwarp();
            if (lane == 0) {
                const float f = __expf(m_old - u);  // exp(-inf) = 0
                s_f[r] = f;
                s_l[r] = s_l[r] * f + l;
                s_m[r] = m;
            }
        }
        __syncthreads();
        const float f0 = s_f[mw * 16 + g], f1 = s_f[mw * 16 + g + 8];
#pragma unroll
        for (int i = 0; i < NT; ++i) {
            o[i][0] *= f0;
            o[i][1] *= f0;
            o[i][2] *= f1;
            o[i][3] *= f1;
        }
#pragma unroll
        for (int kk = 0; kk < kLatentTile / 16; ++kk) {
            uint32_t pa[4];
            ldmatrix_x4(smem_u32(ps) + (uint32_t)(((mw * 16 + (mi & 1) * 8 + mr) * kPPitch + kk * 16 + (mi >> 1) * 8) * 2), pa[0], pa[1],
                        pa[2], pa[3]);
#pragma unroll
            for (int dp = 0; dp < NT / 2; ++dp) {
                const int col = nw * NT * 8 + dp * 16;
                if (col < a.rank_pitch) {  // the same for the whole warp
                    uint32_t b[4];
                    ldmatrix_x4_trans(b, ks + (uint32_t)((kk * 16 + (mi & 1) * 8 + mr) * pitch + (col + (mi >> 1) * 8) * 2));
                    mma_f16_16816(o[2 * dp], pa[0], pa[1], pa[2], pa[3], b[0], b[1]);
                    mma_f16_16816(o[2 * dp + 1], pa[0], pa[1], pa[2], pa[3], b[2], b[3]);
                }
            }
        }
        __syncthreads();  // the buffer is refilled by the copy issued in the next iteration
    }
    const int stride = a.rank_pitch + kLatentPartTail;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int r = mw * 16 + g + 8 * half;
        if (r0 + r >= n_rows) continue;
        float* dst = a.part + ((size_t)(r0 + r) * a.max_splits + split) * stride;
#pragma unroll
        for (int i = 0; i < NT; ++i) {
            const int col = nw * NT * 8 + i * 8 + 2 * tq;
            if (col < a.rank_pitch) *reinterpret_cast<float2*>(dst + col) = make_float2(o[i][2 * half], o[i][2 * half + 1]);
        }
        if (nw == 0 && tq == 0) *reinterpret_cast<float2*>(dst + a.rank_pitch) = make_float2(s_m[r], s_l[r]);
    }
}

template <int MT>
constexpr int latent_mma_smem(int row_width) {
    return (16 * MT + 2 * kLatentTile) * (row_width * 2 + 16) + 16 * MT * ((kLatentTile + 4) * 4 + (kLatentTile + 8) * 2 + 12);
}

// ---- prompt block: the splits of every query row put together, as hi + lo MMA operands of the value GEMM.
// grid: rows; out: [2 planes][kPrefillTokens][heads * in_pitch], in_pitch >= rank_pitch inputs per head
template <typename T>
static __global__ void __launch_bounds__(128) prefill_latent_combine_kernel(const LatentAttnArgs a, int tile_rows, T* out, int in_pitch) {
    __shared__ float wt[kLatentMaxSplits];
    pdl_launch_dependents();
    pdl_wait();
    const int row = blockIdx.x, t = row / a.heads, h = row - t * a.heads;
    const int n_rows = a.n_tokens * a.heads;
    // the row's tile in the attention launch (0 = the kernel that takes one row at a time)
    const int r0 = tile_rows > 0 ? row / tile_rows * tile_rows : row, r1 = tile_rows > 0 ? min(r0 + tile_rows, n_rows) - 1 : row;
    const LatentSpan sp = latent_span(a.start_pos + r0 / a.heads, a.start_pos + r1 / a.heads, a.window, a.max_splits, a.min_chunk);
    const int stride = a.rank_pitch + kLatentPartTail, lane = threadIdx.x & 31;
    const float* p = a.part + (size_t)row * a.max_splits * stride;
    if (threadIdx.x < 32) {
        const bool in = lane < sp.n_eff;
        const float m = in ? __ldcg(p + (size_t)lane * stride + a.rank_pitch) : -INFINITY;
        const float l = in ? __ldcg(p + (size_t)lane * stride + a.rank_pitch + 1) : 0.f;
        const float mm = warp_max(m);
        const float e = in ? __expf(m - mm) : 0.f;
        const float sum = warp_sum(e * l);
        wt[lane] = __fdiv_rn(e, sum);
    }
    __syncthreads();
    T* hi_row = out + (size_t)t * a.heads * in_pitch + (size_t)h * in_pitch;
    T* lo_row = hi_row + (size_t)kPrefillTokens * a.heads * in_pitch;
    for (int k = 2 * threadIdx.x; k < a.rank_pitch; k += 256) {
        float2 v = make_float2(0.f, 0.f);
#pragma unroll 4
        for (int s = 0; s < sp.n_eff; ++s) {
            const float2 x = __ldcg(reinterpret_cast<const float2*>(p + (size_t)s * stride + k));
            v.x = fmaf(wt[s], x.x, v.x);
            v.y = fmaf(wt[s], x.y, v.y);
        }
        T hi[2], lo[2];
        split_pair(v.x, hi[0], lo[0]);
        split_pair(v.y, hi[1], lo[1]);
        hi_row[k] = hi[0];
        hi_row[k + 1] = hi[1];
        lo_row[k] = lo[0];
        lo_row[k + 1] = lo[1];
    }
}

// ---- prompt block: after the input GEMM (partial sums over ranges of K, added in range order): plain queries -> hi + lo
// operands of the query GEMM, rotated parts turned into query and cache rows, latent normed into its cache row, gates
// through the sigmoid.  The section layout of the rows is that of latent_in_rows.
// grid: (tokens, 1 + query sections): y = 0 takes latent, rotated key part and gates, y >= 1 512 query rows each.
constexpr int kLatFinishThreads = 256;
struct PrefillLatentFinishArgs {
    const float* part;  // [splits][kPrefillTokens][n_rows]
    int n_rows, splits;
    int start_pos, seq_len;
    void* qn;           // plain queries: [2 planes][kPrefillTokens][heads * dim_pitch]
    float* gate;        // [kPrefillTokens][heads]
    StepState* st;
    LatentArgs lat;     // query: [kPrefillTokens * heads][row_width]
};
template <typename T>
static __global__ void __launch_bounds__(kLatFinishThreads) prefill_latent_finish_kernel(const PrefillLatentFinishArgs a) {
    extern __shared__ float fin_smem[];  // the raw latent
    __shared__ float red[kLatFinishThreads / 32];
    pdl_launch_dependents();
    pdl_wait();
    const LatentArgs& L = a.lat;
    const int t = blockIdx.x, tid = threadIdx.x, pos = a.start_pos + t;
    if (pos < 0 || pos >= a.seq_len) {
        if (tid == 0) atomicOr(&a.st->status, kStatusBadPos);
        return;
    }
    auto sum2 = [&](int row) -> float2 {
        float2 p[kPfMaxSplits], v = make_float2(0.f, 0.f);
#pragma unroll
        for (int s = 0; s < kPfMaxSplits; ++s)
            if (s < a.splits) p[s] = *reinterpret_cast<const float2*>(a.part + ((size_t)s * kPrefillTokens + t) * a.n_rows + row);
#pragma unroll
        for (int s = 0; s < kPfMaxSplits; ++s)
            if (s < a.splits) {
                v.x += p[s].x;
                v.y += p[s].y;
            }
        return v;
    };
    auto turn = [&](float2 v, int j) -> float2 {
        const float2 cs = __ldg(L.rope + (size_t)pos * (L.rot >> 1) + (j >> 1));
        return make_float2(__fsub_rn(__fmul_rn(v.x, cs.x), __fmul_rn(v.y, cs.y)), __fadd_rn(__fmul_rn(v.y, cs.x), __fmul_rn(v.x, cs.y)));
    };
    const int q_rows = L.q_plain_rows + L.q_rot_rows;
    if (blockIdx.y > 0) {
        const int row = ((int)blockIdx.y - 1) * 2 * kLatFinishThreads + 2 * tid;
        if (row >= q_rows) return;
        float2 v = sum2(row);
        if (row < L.q_plain_rows) {
            T* qn = reinterpret_cast<T*>(a.qn) + (size_t)t * L.heads * L.dim_pitch;
            const size_t plane = (size_t)kPrefillTokens * L.heads * L.dim_pitch;
            const float x[2] = {v.x, v.y};
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int r = row + i;
                if (r >= L.heads * L.dim) continue;
                const size_t at = (size_t)(r / L.dim) * L.dim_pitch + r % L.dim;
                T hi, lo;
                split_pair(x[i], hi, lo);
                qn[at] = hi;
                qn[plane + at] = lo;
            }
        } else {
            const int r = row - L.q_plain_rows, h = r / L.rot, j = r - h * L.rot;
            v = turn(v, j);
            __half* q = reinterpret_cast<__half*>(L.query) + ((size_t)t * L.heads + h) * L.row_width + L.rank_pitch + j;
            *reinterpret_cast<__half2*>(q) = __floats2half2_rn(v.x, v.y);
        }
        return;
    }
    float ss = 0.f;
    for (int r = 2 * tid; r < L.latent_rows; r += 2 * kLatFinishThreads) {
        const float2 v = sum2(q_rows + r);  // a padding row has zero weights
        fin_smem[r] = v.x;
        fin_smem[r + 1] = v.y;
        ss = fmaf(v.x, v.x, fmaf(v.y, v.y, ss));
    }
    __half* crow = reinterpret_cast<__half*>(L.cache) + (size_t)pos * L.row_width;
    for (int j = 2 * tid; j < L.rot; j += 2 * kLatFinishThreads) {
        const float2 v = turn(sum2(q_rows + L.latent_rows + j), j);
        *reinterpret_cast<__half2*>(crow + L.rank_pitch + j) = __floats2half2_rn(v.x, v.y);
    }
    const int gate0 = q_rows + L.latent_rows + L.rot;
    for (int h = 2 * tid; h < L.heads; h += 2 * kLatFinishThreads) {
        const float2 v = sum2(gate0 + h);
        a.gate[(size_t)t * L.heads + h] = sigmoid_f(v.x);
        if (h + 1 < L.heads) a.gate[(size_t)t * L.heads + h + 1] = sigmoid_f(v.y);
    }
    ss = warp_sum(ss);
    if ((tid & 31) == 0) red[tid >> 5] = ss;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int w = 0; w < kLatFinishThreads / 32; ++w) tot += red[w];
    const float scale = __fdiv_rn(1.0f, __fsqrt_rn(__fadd_rn(__fdiv_rn(tot, (float)L.rank), L.norm_eps)));
    for (int r = tid; r < L.rank; r += kLatFinishThreads)
        crow[r] = __float2half_rn(__fmul_rn(__fmul_rn(fin_smem[r], scale), __ldg(L.norm_w + r)));
}

}  // namespace lpp
