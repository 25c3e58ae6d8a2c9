// Attention over shared rows: one cache row per position serves as key and, with its first rank_pitch columns, as value.
// Latent attention (latent.cuh) has one such row for all heads, attention whose values are its unrotated keys
// (shared_kv.cuh) one per key/value head.  Also the two small kernels around latent attention on the batched prompt path.
//
// Heads that share a row form a group.  The query rows of a group in an attention launch are its (token, head) pairs,
// row = token * heads + head: one row block for a decode step, n_tokens x heads rows for a prompt block.  A CTA takes a
// tile of query rows and one of the splits of the keys that the tile's tokens can see (sliding window; a tile's tokens
// are neighbours, so their windows nearly coincide) and writes the unnormalised weighted sum, its maximum and its sum.
// Whoever consumes the result puts the splits together: the value GEMV of latent attention when decoding, the last CTA
// of a row tile to finish when `out` is set, prefill_latent_combine_kernel in a prompt block.
#pragma once
#include "latent.cuh"
#include "prefill.cuh"

namespace lpp {

struct LatentAttnArgs {
    const void* q;      // [token][all_heads][row_width]
    const void* cache;  // [group][positions][row_width], this layer's
    float* part;        // [token][all_heads][max_splits][rank_pitch + kLatentPartTail]
    const StepState* st;
    int start_pos;      // position of token 0; < 0 = the step's device-resident position
    int n_tokens;
    int heads;          // query heads of a group: they share its cache rows
    int all_heads;      // heads x groups
    int score_skip;     // 16-column steps at the start of a row that scores leave out (zero in the queries)
    int rank_pitch, row_width;
    int window, max_splits, min_chunk;
    int seq_len;
    float scale;
    float softcap;      // > 0: a score s becomes softcap * tanh(s / softcap)
    float cap_rate;     // 2 / softcap
    // One token, splits put together by the CTA that finishes last: out[head * out_cols + col] = result * gate
    float* out;              // nullptr = partial results stay in `part`
    const float* gate;       // [all_heads * out_cols], prompt blocks [token][all_heads * out_cols]; nullptr = none
    int out_cols;            // valid columns of a result
    unsigned int* counters;  // one per row tile (or head), zero between launches
    // Tensor-core kernel: the splits of a row tile form a cluster and put themselves together
    int cluster;             // 0 = partial results to `part`
    // A prompt block's finished rows, hi + lo: [2 planes][kPrefillTokens][plane_row], head after head of plane_pitch
    // columns, of which the first plane_cols are written
    __nv_bfloat16* planes;
    int plane_pitch, plane_cols, plane_row;
};

// Global query row of a group's row r.
__device__ __forceinline__ int latent_row(const LatentAttnArgs& a, int group, int r) {
    const int t = r / a.heads;
    return t * a.all_heads + group * a.heads + (r - t * a.heads);
}
// softcap * tanh(s / softcap) as softcap - 2 softcap / (1 + exp(2 s / softcap)): an absolute error of a few 1e-7 softcap.
__device__ __forceinline__ float capped_score(const LatentAttnArgs& a, float s) {
    return a.softcap - __fdividef(2.f * a.softcap, 1.f + __expf(s * a.cap_rate));
}
// The last of `n` CTAs to get here returns true, with the others' global stores visible.  Called by all threads of the CTA; the
// barriers put every thread's accesses before and after the counter's release and acquire.
__device__ __forceinline__ bool latent_last_arrival(unsigned int* counter, unsigned int n, int* flag, int tid) {
    __syncthreads();
    if (tid == 0) {
        unsigned int ticket;
        asm volatile("atom.add.acq_rel.gpu.global.u32 %0, [%1], 1;" : "=r"(ticket) : "l"(counter) : "memory");
        *flag = ticket == n - 1u;
        if (ticket == n - 1u) *counter = 0u;
    }
    __syncthreads();
    return *flag;
}
__device__ __forceinline__ void latent_out(const LatentAttnArgs& a, int head, int col, float v) {
    const int at = head * a.out_cols + col;
    a.out[at] = a.gate ? v * __ldcg(a.gate + at) : v;
}
__device__ __forceinline__ void latent_out4(const LatentAttnArgs& a, int head, int col, float4 v) {
    const int at = head * a.out_cols + col;
    if ((a.out_cols & 3) == 0) {
        if (col >= a.out_cols) return;
        if (a.gate) {
            const float4 g = __ldcg(reinterpret_cast<const float4*>(a.gate + at));
            v.x *= g.x; v.y *= g.y; v.z *= g.z; v.w *= g.w;
        }
        *reinterpret_cast<float4*>(a.out + at) = v;
        return;
    }
    const float y[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int c = 0; c < 4; ++c)
        if (col + c < a.out_cols) latent_out(a, head, col + c, y[c]);
}
constexpr int kLatentMaxCluster = 8;
constexpr int kLatentTile = 64;        // keys per shared-memory tile
constexpr int kLatentThreads = 256;

// Heads `head` .. head + n - 1 of a token from their n_eff partial results: added up in split order and finished.  NT threads;
// scratch: n * kLatentMaxSplits + 4 NT floats.  A thread takes four columns of a head and, where there are threads to
// spare, half of the splits.  Kept short: this code is fetched by a few CTAs at the end of every launch.
template <int NT>
__device__ __forceinline__ void latent_combine_heads(const LatentAttnArgs& a, int head, int n, int n_eff, float* scratch, int tid) {
    float* wt = scratch;                                                       // [n][kLatentMaxSplits]
    float4* half = reinterpret_cast<float4*>(scratch + n * kLatentMaxSplits);  // [NT]
    const int stride = a.rank_pitch + kLatentPartTail, warp = tid >> 5, lane = tid & 31;
    const int q4 = a.rank_pitch >> 2, slots = n * q4;
    const int halves = 2 * slots <= NT ? 2 : 1, per = NT / halves, part = tid >= per ? 1 : 0;
    const int s_half = halves == 2 ? (n_eff + 1) >> 1 : n_eff, s_begin = part ? s_half : 0, s_end = part ? n_eff : s_half;
    const float* p0 = a.part + (size_t)head * a.max_splits * stride;
    // weights of the splits: exp(m_s - max m) / sum of l
    auto weights = [&]() {
        for (int k = warp; k < n; k += NT / 32) {
            const float2 ml = lane < n_eff ? __ldcg(reinterpret_cast<const float2*>(p0 + ((size_t)k * a.max_splits + lane) * stride + a.rank_pitch))
                                           : make_float2(-INFINITY, 0.f);
            const float e = expf(ml.x - warp_max(ml.x));
            wt[k * kLatentMaxSplits + lane] = __fdiv_rn(e, warp_sum(e * ml.y));
        }
        __syncthreads();
    };
    for (int base = 0; base < slots; base += per) {
        const int slot = min(base + tid - part * per, slots - 1), r = slot / q4, col = (slot - r * q4) << 2;
        const bool mine = base + tid - part * per < slots;
        const float* p = p0 + (size_t)r * a.max_splits * stride + col;
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int s0 = s_begin, first = base == 0; s0 < s_end || first; s0 += 8, first = 0) {
            float4 v[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) v[i] = __ldcg(reinterpret_cast<const float4*>(p + (size_t)min(s0 + i, n_eff - 1) * stride));
            if (first) weights();  // beside the first loads
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const float w = s0 + i < s_end ? wt[r * kLatentMaxSplits + s0 + i] : 0.f;
                acc.x = fmaf(w, v[i].x, acc.x); acc.y = fmaf(w, v[i].y, acc.y); acc.z = fmaf(w, v[i].z, acc.z); acc.w = fmaf(w, v[i].w, acc.w);
            }
        }
        if (halves == 2) {
            half[tid] = acc;
            __syncthreads();
            if (part) return;
            const float4 b = half[tid + per];
            acc.x += b.x; acc.y += b.y; acc.z += b.z; acc.w += b.w;
        }
        if (!mine) continue;
        latent_out4(a, head + r, col, acc);
    }
}

// ---- any sizes, FP32 or FP16 rows, FP32 arithmetic.  grid: (splits, heads, tokens)
constexpr int kLatentMaxPerThread = 8;  // latent elements of one thread: ranks up to 2048
template <typename KT>
static __global__ void __launch_bounds__(kLatentThreads) latent_attn_kernel(const LatentAttnArgs a) {
    extern __shared__ __align__(16) float lat_smem[];  // query row, then scores of a tile
    __shared__ float s_f, s_m, s_l;
    __shared__ int s_last;
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
    const size_t row = (size_t)blockIdx.z * a.all_heads + blockIdx.y;
    const KT* q = reinterpret_cast<const KT*>(a.q) + row * a.row_width;
    const KT* kc = reinterpret_cast<const KT*>(a.cache) + (size_t)(blockIdx.y / a.heads) * a.seq_len * a.row_width;
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
            if (lane == 0) sc[k] = a.softcap > 0.f ? a.softcap * tanhf(__fdiv_rn(s * a.scale, a.softcap)) : s * a.scale;
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
    if (a.out && sp.n_eff == 1) {  // all keys seen
#pragma unroll
        for (int j = 0; j < kLatentMaxPerThread; ++j)
            if (tid + j * kLatentThreads < a.out_cols) latent_out(a, blockIdx.y, tid + j * kLatentThreads, __fdiv_rn(o[j], s_l));
        return;
    }
    float* p = a.part + (row * a.max_splits + split) * (a.rank_pitch + kLatentPartTail);
#pragma unroll
    for (int j = 0; j < kLatentMaxPerThread; ++j)
        if (tid + j * kLatentThreads < a.rank_pitch) p[tid + j * kLatentThreads] = o[j];
    if (tid == 0) {
        p[a.rank_pitch] = s_m;
        p[a.rank_pitch + 1] = s_l;
    }
    if (!a.out || !latent_last_arrival(a.counters + blockIdx.y, sp.n_eff, &s_last, tid)) return;
    latent_combine_heads<kLatentThreads>(a, blockIdx.y, 1, sp.n_eff, lat_smem, tid);
}

// ---- tensor cores, FP16 rows.  grid: (splits, row tiles of 16 MT, groups); with `cluster` set the splits of a row tile are one
// thread-block cluster.
//
// Query tile and 64-key tiles (double buffered, 16-byte asynchronous copies) lie in shared memory in rows padded by 16
// bytes.  Per tile: scores by mma.sync m16n8k16, the NW warps taking 16 keys (four groups) and one of NW / 4 parts of the row
// width each, the parts to shared memory (FP32); sum of the parts, mask, running maximum, exponentials and sum in FP32, a
// few rows per warp; probabilities (FP16) times the latent part of the same tile, every warp holding all query rows of
// NT * 8 columns of the result.  Every key row is read from shared memory once per product, the query tile four times.
//
// The splits meet in one of two ways.  Prompt block: every CTA leaves its unnormalised result in its own shared memory, and
// after a cluster barrier each adds up a share of the row tile over all CTAs through distributed shared memory; the
// finished rows go out as hi + lo operands.  One token: partial results to part, as the CUDA-core kernel does (for 17
// splits of 64 keys the cluster's gang launch and two barriers cost 4 us more than the value GEMV needs to add them up);
// with `out` set the last CTA of a row tile puts them together, and a span of one split goes out at once.
__device__ __forceinline__ void cluster_barrier() {
    asm volatile("barrier.cluster.arrive.release;\n\tbarrier.cluster.wait.acquire;" ::: "memory");
}
__device__ __forceinline__ uint32_t cluster_map(uint32_t smem_addr, uint32_t rank) {
    uint32_t r;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(smem_addr), "r"(rank));
    return r;
}
// (volatile keeps these between the barriers, which are volatile too; no memory clobber, so several are in flight at once)
__device__ __forceinline__ float4 cluster_load4(uint32_t addr) {
    float4 v;
    asm volatile("ld.shared::cluster.v4.f32 {%0,%1,%2,%3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(addr));
    return v;
}
__device__ __forceinline__ float cluster_load(uint32_t addr) {
    float v;
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr));
    return v;
}

// Columns col .. col + 3 of a finished row of a prompt block, times the gate, as hi + lo operands.
template <bool GATED>
__device__ __forceinline__ void latent_planes4(const LatentAttnArgs& a, int t, int h, int col, float (&y)[4]) {
    if (GATED && a.gate) {
        const float* g = a.gate + ((size_t)t * a.all_heads + h) * a.plane_cols + col;
#pragma unroll
        for (int c = 0; c < 4; ++c)
            if (col + c < a.plane_cols) y[c] *= __ldcg(g + c);
    }
    __nv_bfloat16* d = a.planes + (size_t)t * a.plane_row + (size_t)h * a.plane_pitch + col;
    __nv_bfloat16* d_lo = d + (size_t)kPrefillTokens * a.plane_row;
    __align__(8) __nv_bfloat16 hi[4], lo[4];
#pragma unroll
    for (int c = 0; c < 4; ++c) split_pair(y[c], hi[c], lo[c]);
    if (!GATED || ((a.plane_pitch | a.plane_cols) & 3) == 0) {  // (rows of latents are padded)
        if (col < a.plane_cols) {
            *reinterpret_cast<uint2*>(d) = *reinterpret_cast<const uint2*>(hi);
            *reinterpret_cast<uint2*>(d_lo) = *reinterpret_cast<const uint2*>(lo);
        }
    } else {
#pragma unroll
        for (int c = 0; c < 4; ++c)
            if (col + c < a.plane_cols) d[c] = hi[c], d_lo[c] = lo[c];
    }
}

constexpr int kLatScPitch = kLatentTile + 4, kLatPPitch = kLatentTile + 8;
template <int MT, int NW>
constexpr int latent_mma_smem(int row_width) {
    return (16 * MT + 2 * kLatentTile) * (row_width * 2 + 16) + 16 * MT * (NW / 4 * kLatScPitch * 4 + kLatPPitch * 2 + 12 + kLatentMaxCluster * 4);
}

// SKV: attention of shared_kv.cuh (groups, score cap, gates, `out`); an argument because latent attention should not fetch its
// code.
template <int MT, int NT, int NW, bool SKV>
static __global__ void __launch_bounds__(NW * 32) latent_attn_mma_kernel(const LatentAttnArgs a) {
    constexpr int kRows = 16 * MT, kThreads = NW * 32, kParts = NW / 4, kRowsPerWarp = kRows / NW;
    static_assert(NT % 2 == 0, "column tiles go in pairs");
    static_assert(NW % 4 == 0 && kRows % NW == 0, "warps share the rows evenly");
    extern __shared__ __align__(128) unsigned char lm_smem[];
    const int pitch = a.row_width * 2 + 16;
    unsigned char* qs = lm_smem;
    unsigned char* kt = qs + kRows * pitch;
    float* sc = reinterpret_cast<float*>(kt + 2 * kLatentTile * pitch);          // [kParts][kRows][kLatScPitch]
    __half* ps = reinterpret_cast<__half*>(sc + kParts * kRows * kLatScPitch);  // [kRows][kLatPPitch]
    float* s_m = reinterpret_cast<float*>(ps + kRows * kLatPPitch);
    float* s_l = s_m + kRows;
    float* s_f = s_l + kRows;
    float* s_w = s_f + kRows;  // [kRows][kLatentMaxCluster] weights of the cluster's CTAs
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
    const bool active = split < sp.n_eff;
    if (!active && !a.cluster) {
        pdl_wait();
        return;
    }
    const int k_begin = sp.first + split * sp.chunk, k_end = min(k_begin + sp.chunk, base + t_hi + 1);
    const int n_tiles = active ? (k_end - k_begin + kLatentTile - 1) / kLatentTile : 0;
    const size_t row_bytes = (size_t)a.row_width * 2;
    const int group = SKV ? blockIdx.z : 0;
    auto row_of = [&](int r) -> int { return SKV ? latent_row(a, group, r) : r; };  // global row of the group's row r
    auto score = [&](float dot) -> float {
        const float s = dot * a.scale;
        return SKV && a.softcap > 0.f ? capped_score(a, s) : s;
    };
    const unsigned char* cache = reinterpret_cast<const unsigned char*>(a.cache) + (size_t)group * a.seq_len * row_bytes;
    const int pieces = a.row_width / 8;

    // rows of the tile in [lo, hi); with `fill` the rows between k_end and the next multiple of 16 become zero
    auto load_keys = [&](int tile, int lo, int hi, bool fill) {
        unsigned char* dst = kt + (size_t)(tile & 1) * kLatentTile * pitch;
        const int p0 = k_begin + tile * kLatentTile;
        const int rows = min(kLatentTile, (k_end - p0 + 15) & ~15);
        for (int r = warp; r < rows; r += NW) {
            const int p = p0 + r;
            const bool in = p >= lo && p < hi;
            if (!in && !(fill && p >= k_end)) continue;
            const unsigned char* src = in ? cache + (size_t)p * row_bytes : cache;
            for (int col = lane; col < pieces; col += 32) cp_async_16(dst + r * pitch + col * 16, src + (in ? col * 16 : 0), in);
        }
    };
    // cache rows of earlier steps and blocks do not depend on the preceding kernels
    if (active) load_keys(0, k_begin, min(k_end, base), false);
    pdl_wait();
    if (active) {
        load_keys(0, max(k_begin, base), k_end, true);
        for (int r = warp; r < kRows; r += NW) {
            const bool in = r0 + r < n_rows;
            const unsigned char* src = reinterpret_cast<const unsigned char*>(a.q) + (in ? (size_t)row_of(r0 + r) * row_bytes : 0);
            for (int col = lane; col < pieces; col += 32) cp_async_16(qs + r * pitch + col * 16, src + (in ? col * 16 : 0), in);
        }
    }
    cp_async_commit();
    if (tid < kRows) {
        s_m[tid] = -INFINITY;
        s_l[tid] = 0.f;
    }

    const int g = lane >> 2, tq = lane & 3, mi = lane >> 3, mr = lane & 7;
    float o[MT][NT][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int i = 0; i < NT; ++i) o[m][i][0] = o[m][i][1] = o[m][i][2] = o[m][i][3] = 0.f;
    const int skip = SKV ? a.score_skip : 0, k_steps = a.row_width / 16 - skip;
    const int key16 = warp & 3, part = warp >> 2;  // scores: this warp's 16 keys and its share of the k-steps
    const int ks0 = skip + part * k_steps / kParts, ks1 = skip + (part + 1) * k_steps / kParts;
    const uint32_t q_addr = smem_u32(qs) + (uint32_t)(((mi & 1) * 8 + mr) * pitch + (mi >> 1) * 16);
    const uint32_t p_addr = smem_u32(ps) + (uint32_t)((((mi & 1) * 8 + mr) * kLatPPitch + (mi >> 1) * 8) * 2);

    for (int tile = 0; tile < n_tiles; ++tile) {
        cp_async_wait<0>();
        __syncthreads();  // this tile is here, and nobody reads the other buffer any more
        if (tile + 1 < n_tiles) {
            load_keys(tile + 1, k_begin, k_end, true);
            cp_async_commit();
        }
        const uint32_t ks = smem_u32(kt) + (uint32_t)((tile & 1) * kLatentTile * pitch);
        const int p0 = k_begin + tile * kLatentTile;
        const int groups = min(kLatentTile / 16, (k_end - p0 + 15) >> 4);  // 16-key groups with keys in them
        if (key16 < groups) {
            float c[MT][2][4];
#pragma unroll
            for (int m = 0; m < MT; ++m)
#pragma unroll
                for (int j = 0; j < 2; ++j) c[m][j][0] = c[m][j][1] = c[m][j][2] = c[m][j][3] = 0.f;
            const uint32_t b_addr = ks + (uint32_t)((key16 * 16 + (mi >> 1) * 8 + mr) * pitch + (mi & 1) * 16);
#pragma unroll 3
            for (int kk = ks0; kk < ks1; ++kk) {
                uint32_t b[4], qa[MT][4];
                ldmatrix_x4(b_addr + (uint32_t)kk * 32u, b[0], b[1], b[2], b[3]);
#pragma unroll
                for (int m = 0; m < MT; ++m)
                    ldmatrix_x4(q_addr + (uint32_t)(m * 16 * pitch) + (uint32_t)kk * 32u, qa[m][0], qa[m][1], qa[m][2], qa[m][3]);
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    mma_f16_16816(c[m][0], qa[m][0], qa[m][1], qa[m][2], qa[m][3], b[0], b[1]);
                    mma_f16_16816(c[m][1], qa[m][0], qa[m][1], qa[m][2], qa[m][3], b[2], b[3]);
                }
            }
#pragma unroll
            for (int m = 0; m < MT; ++m)
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    float* d = sc + (part * kRows + m * 16 + g) * kLatScPitch + key16 * 16 + j * 8 + 2 * tq;
                    *reinterpret_cast<float2*>(d) = make_float2(c[m][j][0], c[m][j][1]);
                    *reinterpret_cast<float2*>(d + 8 * kLatScPitch) = make_float2(c[m][j][2], c[m][j][3]);
                }
        }
        __syncthreads();
        {  // mask and online softmax: kRowsPerWarp rows per warp, two keys per lane
            const int p = p0 + lane;
            float x0[kRowsPerWarp], x1[kRowsPerWarp], m_old[kRowsPerWarp], m_new[kRowsPerWarp], l[kRowsPerWarp];
#pragma unroll
            for (int i = 0; i < kRowsPerWarp; ++i) {
                const int r = warp * kRowsPerWarp + i;
                const int last = base + min(r0 + r, n_rows - 1) / a.heads, lo = a.window > 0 ? last - a.window + 1 : 0;
                const float* s0 = sc + r * kLatScPitch + lane;
                float v0 = 0.f, v1 = 0.f;
#pragma unroll
                for (int q = 0; q < kParts; ++q) {
                    v0 += s0[q * kRows * kLatScPitch];
                    v1 += s0[q * kRows * kLatScPitch + 32];
                }
                x0[i] = (p >= lo && p <= last && p < k_end) ? score(v0) : -INFINITY;
                x1[i] = (p + 32 >= lo && p + 32 <= last && p + 32 < k_end) ? score(v1) : -INFINITY;
                m_old[i] = s_m[r];
                m_new[i] = fmaxf(x0[i], x1[i]);
            }
#pragma unroll
            for (int i = 0; i < kRowsPerWarp; ++i) m_new[i] = fmaxf(m_old[i], warp_max(m_new[i]));
#pragma unroll
            for (int i = 0; i < kRowsPerWarp; ++i) {
                const float u = m_new[i] == -INFINITY ? 0.f : m_new[i];  // nothing visible to this row yet
                x0[i] = __expf(x0[i] - u);
                x1[i] = __expf(x1[i] - u);
                m_old[i] = __expf(m_old[i] - u);  // what earlier tiles are rescaled by; exp(-inf) = 0
                l[i] = x0[i] + x1[i];
            }
#pragma unroll
            for (int i = 0; i < kRowsPerWarp; ++i) l[i] = warp_sum(l[i]);
#pragma unroll
            for (int i = 0; i < kRowsPerWarp; ++i) {
                const int r = warp * kRowsPerWarp + i;
                ps[r * kLatPPitch + lane] = __float2half_rn(x0[i]);
                ps[r * kLatPPitch + lane + 32] = __float2half_rn(x1[i]);
                if (lane == 0) {
                    s_f[r] = m_old[i];
                    s_l[r] = s_l[r] * m_old[i] + l[i];
                    s_m[r] = m_new[i];
                }
            }
        }
        __syncthreads();
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            const float f0 = s_f[m * 16 + g], f1 = s_f[m * 16 + g + 8];
#pragma unroll
            for (int i = 0; i < NT; ++i) {
                o[m][i][0] *= f0;
                o[m][i][1] *= f0;
                o[m][i][2] *= f1;
                o[m][i][3] *= f1;
            }
        }
#pragma unroll
        for (int kk = 0; kk < kLatentTile / 16; ++kk) {
            if (kk >= groups) break;
            uint32_t pa[MT][4];
#pragma unroll
            for (int m = 0; m < MT; ++m)
                ldmatrix_x4(p_addr + (uint32_t)((m * 16 * kLatPPitch + kk * 16) * 2), pa[m][0], pa[m][1], pa[m][2], pa[m][3]);
#pragma unroll
            for (int dp = 0; dp < NT / 2; ++dp) {
                const int col = warp * NT * 8 + dp * 16;
                if (col < a.rank_pitch) {  // the same for the whole warp
                    uint32_t b[4];
                    ldmatrix_x4_trans(b, ks + (uint32_t)((kk * 16 + (mi & 1) * 8 + mr) * pitch + (col + (mi >> 1) * 8) * 2));
#pragma unroll
                    for (int m = 0; m < MT; ++m) {
                        mma_f16_16816(o[m][2 * dp], pa[m][0], pa[m][1], pa[m][2], pa[m][3], b[0], b[1]);
                        mma_f16_16816(o[m][2 * dp + 1], pa[m][0], pa[m][1], pa[m][2], pa[m][3], b[2], b[3]);
                    }
                }
            }
        }
    }
    __syncthreads();
    if (!a.cluster) {
        if (SKV && a.out && sp.n_eff == 1) {  // all keys seen: finished rows
#pragma unroll
            for (int m = 0; m < MT; ++m)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int r = m * 16 + g + 8 * half;
                    if (r0 + r >= n_rows) continue;
                    const int head = group * a.heads + r0 + r;  // one token
                    const float l = s_l[r];
#pragma unroll
                    for (int i = 0; i < NT; ++i) {
                        const int col = warp * NT * 8 + i * 8 + 2 * tq;
                        if (col < a.out_cols) latent_out(a, head, col, __fdiv_rn(o[m][i][2 * half], l));
                        if (col + 1 < a.out_cols) latent_out(a, head, col + 1, __fdiv_rn(o[m][i][2 * half + 1], l));
                    }
                }
            return;
        }
        const int stride = a.rank_pitch + kLatentPartTail;
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int r = m * 16 + g + 8 * half;
                if (r0 + r >= n_rows) continue;
                float* dst = a.part + ((size_t)row_of(r0 + r) * a.max_splits + split) * stride;
#pragma unroll
                for (int i = 0; i < NT; ++i) {
                    const int col = warp * NT * 8 + i * 8 + 2 * tq;
                    if (col < a.rank_pitch) *reinterpret_cast<float2*>(dst + col) = make_float2(o[m][i][2 * half], o[m][i][2 * half + 1]);
                }
                if (warp == 0 && tq == 0) *reinterpret_cast<float2*>(dst + a.rank_pitch) = make_float2(s_m[r], s_l[r]);
            }
        if constexpr (SKV) {
            // scratch over the scores, whose space is larger: [kParts][kRows][kLatScPitch] floats
            static_assert(MT > 1 || kParts * kRows * kLatScPitch >= kRows * kLatentMaxSplits + 4 * kThreads, "scratch of the combination");
            if (MT == 1 && a.out && latent_last_arrival(a.counters + group * gridDim.y + blockIdx.y, sp.n_eff, reinterpret_cast<int*>(s_w), tid))
                latent_combine_heads<kThreads>(a, group * a.heads + r0, min(kRows, n_rows - r0), sp.n_eff, sc, tid);
        }
        return;
    }
    // this CTA's result over the key tiles (nobody reads them any more), rows of rank_pitch + 4 floats: that fits, as
    // 16 MT rows of 4 bytes are no more than 2 x 64 rows of 2 bytes
    float* os = reinterpret_cast<float*>(kt);
    const int o_pitch = a.rank_pitch + 4;
    if (active) {
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                float* dst = os + (m * 16 + g + 8 * half) * o_pitch;
#pragma unroll
                for (int i = 0; i < NT; ++i) {
                    const int col = warp * NT * 8 + i * 8 + 2 * tq;
                    if (col < a.rank_pitch) *reinterpret_cast<float2*>(dst + col) = make_float2(o[m][i][2 * half], o[m][i][2 * half + 1]);
                }
            }
    }
    cluster_barrier();
    const int n_cta = gridDim.x, n_eff = sp.n_eff;
    // weights of the CTAs, eight lanes per row: exp(m_c - max m) / sum of l
    for (int i = tid; i < kRows * kLatentMaxCluster; i += kThreads) {
        const int r = i / kLatentMaxCluster, c = i % kLatentMaxCluster;
        float m = -INFINITY, l = 0.f;
        if (c < n_eff) {
            m = cluster_load(cluster_map(smem_u32(s_m + r), c));
            l = cluster_load(cluster_map(smem_u32(s_l + r), c));
        }
        float mm = m;
#pragma unroll
        for (int d = kLatentMaxCluster / 2; d > 0; d >>= 1) mm = fmaxf(mm, __shfl_xor_sync(0xffffffffu, mm, d));
        const float e = c < n_eff ? __expf(m - mm) : 0.f;
        float sum = e * l;
#pragma unroll
        for (int d = kLatentMaxCluster / 2; d > 0; d >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, d);
        s_w[i] = __fdiv_rn(e, sum);
    }
    __syncthreads();
    const int q4 = a.rank_pitch >> 2, rows_here = min(kRows, n_rows - r0);
    for (int i = split * kThreads + tid; i < rows_here * q4; i += n_cta * kThreads) {
        const int r = i / q4, col = (i - r * q4) << 2;
        const uint32_t at = smem_u32(os + r * o_pitch + col);
        float4 x[kLatentMaxCluster];
        float y[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int c = 0; c < kLatentMaxCluster; ++c)
            if (c < n_eff) x[c] = cluster_load4(cluster_map(at, c));
#pragma unroll
        for (int c = 0; c < kLatentMaxCluster; ++c)
            if (c < n_eff) {
                const float w = s_w[r * kLatentMaxCluster + c];
                y[0] = fmaf(w, x[c].x, y[0]); y[1] = fmaf(w, x[c].y, y[1]); y[2] = fmaf(w, x[c].z, y[2]); y[3] = fmaf(w, x[c].w, y[3]);
            }
        const int t = (r0 + r) / a.heads, h = (SKV ? group * a.heads : 0) + (r0 + r - t * a.heads);
        latent_planes4<SKV>(a, t, h, col, y);
    }
    cluster_barrier();  // every CTA's shared memory stays until all have read it
}

// ---- prompt block: the splits of every query row put together (plane_cols columns).  grid: rows
static __global__ void __launch_bounds__(128) prefill_latent_combine_kernel(const LatentAttnArgs a, int tile_rows) {
    __shared__ float wt[kLatentMaxSplits];
    pdl_launch_dependents();
    pdl_wait();
    const int row = blockIdx.x, t = row / a.all_heads, h = row - t * a.all_heads;
    const int n_rows = a.n_tokens * a.heads, r = t * a.heads + h % a.heads;  // of the head's group
    const int r0 = r / tile_rows * tile_rows, r1 = min(r0 + tile_rows, n_rows) - 1;  // the row's tile in the attention launch
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
    for (int k = 4 * threadIdx.x; k < a.rank_pitch; k += 512) {
        float y[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
        for (int s = 0; s < sp.n_eff; ++s) {
            const float4 x = __ldcg(reinterpret_cast<const float4*>(p + (size_t)s * stride + k));
            y[0] = fmaf(wt[s], x.x, y[0]); y[1] = fmaf(wt[s], x.y, y[1]); y[2] = fmaf(wt[s], x.z, y[2]); y[3] = fmaf(wt[s], x.w, y[3]);
        }
        latent_planes4<true>(a, t, h, k, y);
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
