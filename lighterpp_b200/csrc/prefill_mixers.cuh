// What the batched prompt path runs between the GEMMs of a selective-scan layer and of attention whose values are its keys.
#pragma once
#include "mamba.cuh"
#include "prefill.cuh"
#include "shared_kv.cuh"

namespace lpp {

// The sum, in range order, of the partial sums of two neighbouring rows (n_rows apart: tokens, kPrefillTokens apart: ranges).
__device__ __forceinline__ float2 prefill_sum2(const float* part, int n_rows, int splits, int t, int row) {
    float2 p[kPfMaxSplits], v = make_float2(0.f, 0.f);
#pragma unroll
    for (int s = 0; s < kPfMaxSplits; ++s)
        if (s < splits) p[s] = *reinterpret_cast<const float2*>(part + ((size_t)s * kPrefillTokens + t) * n_rows + row);
#pragma unroll
    for (int s = 0; s < kPfMaxSplits; ++s)
        if (s < splits) {
            v.x += p[s].x;
            v.y += p[s].y;
        }
    return v;
}

// ---- attention whose values are its keys (shared_kv.cuh): after the input GEMM (partial sums over ranges of K, added in
// range order), one row pair per thread.
// grid: (tokens, ceil(row pairs / 256))
struct PrefillSharedKvArgs {
    const float* part;  // [splits][kPrefillTokens][n_rows]
    int n_rows, splits;
    int start_pos, seq_len;
    int keys_only;      // only the cache rows are wanted
    StepState* st;
    SharedKvArgs kv;    // query: [kPrefillTokens][heads][row_width] FP16, gate: [kPrefillTokens][heads * dim]
};
static __global__ void __launch_bounds__(256) prefill_shared_kv_finish_kernel(const PrefillSharedKvArgs a) {
    pdl_launch_dependents();
    const SharedKvArgs& s = a.kv;
    const int t = blockIdx.x, row = 2 * ((int)blockIdx.y * 256 + (int)threadIdx.x), pos = a.start_pos + t;
    const bool pos_ok = pos >= 0 && pos < a.seq_len;
    const bool mine = row < a.n_rows && pos_ok && !(a.keys_only && (row < s.q_rows || row >= s.q_rows + s.k_rows));
    RowPrep p0, p1;
    if (mine) {  // constants: ahead of the dependency wait
        p0 = shared_kv_prep(s, pos, row);
        p1 = shared_kv_prep(s, pos, row + 1);
    }
    pdl_wait();
    if (!pos_ok && threadIdx.x == 0) atomicOr(&a.st->status, kStatusBadPos);
    if (!mine) return;
    const float2 v = prefill_sum2(a.part, a.n_rows, a.splits, t, row);
    void* query = reinterpret_cast<__half*>(s.query) + (size_t)t * s.heads * s.row_width;
    float* gate = s.gate + (size_t)t * s.heads * s.dim;
    shared_kv_row(s, query, gate, a.seq_len, pos, row, v.x, v.y, p0);
    shared_kv_row(s, query, gate, a.seq_len, pos, row + 1, v.y, v.x, p1);
}

// ---- selective scan (mamba.cuh)

// Convolution of a prompt block after the input GEMM (partial sums added in range order): x convolved, as FP32 rows and as
// hi + lo operands of the next GEMM; z through the silu.  The inputs of the last taps - 1 tokens go to `tail`; the scan
// copies them to the ring once every CTA of this launch has read it.  A thread takes four channels of kConvTokens tokens;
// TAPS = the number of taps (inputs in registers), or 0 = any (inputs in shared memory).
// grid: (ceil(inner / 256), ceil(tokens / kConvTokens), 2: x, z); shared memory (TAPS 0): (kConvTokens + taps - 1) * 256 floats
constexpr int kConvThreads = 64, kConvTokens = 4;
struct MambaConvArgs {
    const float* part;  // [splits][kPrefillTokens][2 * inner_rows]
    int splits, n_tokens, start_pos, seq_len;
    int inner, inner_rows, taps;
    const float *conv_w, *conv_b;
    const float* ring;
    float *tail, *x, *z;    // x, z: [kPrefillTokens][x_pitch]
    int x_pitch;
    __nv_bfloat16* planes;  // [2 planes][kPrefillTokens][x_pitch]
    StepState* st;
};
// N tokens' sums of the partial sums of rows row .. row + 3, tokens t0 .. (clamped to the block: no branches, so the loads of
// a range of K are in flight together), in range order.
template <int N>
__device__ __forceinline__ void prefill_sums(const float* part, int n_rows, int splits, int n_tokens, int t0, int row, float4 (&v)[N]) {
    const float4* p[N];
#pragma unroll
    for (int i = 0; i < N; ++i) {
        p[i] = reinterpret_cast<const float4*>(part + (size_t)min(max(t0 + i, 0), n_tokens - 1) * n_rows + row);
        v[i] = *p[i];
    }
#pragma unroll 2
    for (int s = 1; s < splits; ++s)
#pragma unroll
        for (int i = 0; i < N; ++i) {
            const float4 w = p[i][(size_t)s * kPrefillTokens * n_rows / 4];
            v[i].x += w.x; v[i].y += w.y; v[i].z += w.z; v[i].w += w.w;
        }
}
// With the fast exponential and division, like the gated feed-forward's activation on this path.
__device__ __forceinline__ float4 silu4(const float4& v) {
    return make_float4(__fdividef(v.x, 1.f + __expf(-v.x)), __fdividef(v.y, 1.f + __expf(-v.y)), __fdividef(v.z, 1.f + __expf(-v.z)),
                       __fdividef(v.w, 1.f + __expf(-v.w)));
}
__device__ __forceinline__ float4 fma4(const float4& a, const float4& b, const float4& c) {
    return make_float4(fmaf(a.x, b.x, c.x), fmaf(a.y, b.y, c.y), fmaf(a.z, b.z, c.z), fmaf(a.w, b.w, c.w));
}
template <int TAPS>
static __global__ void __launch_bounds__(kConvThreads) mamba_conv_kernel(const MambaConvArgs a) {
    extern __shared__ float4 cv_in[];  // [kConvTokens + taps - 1][kConvThreads]; a thread reads back only what it wrote
    pdl_launch_dependents();
    const int tid = threadIdx.x, c = 4 * ((int)blockIdx.x * kConvThreads + tid);
    const int t0 = blockIdx.y * kConvTokens, n_rows = 2 * a.inner_rows, slots = TAPS > 0 ? TAPS - 1 : a.taps - 1;
    const bool in = c < a.inner, ok = a.start_pos >= 0 && a.start_pos + a.n_tokens <= a.seq_len;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    float4 w[TAPS > 0 ? TAPS : 1], bias = zero;
    if (in && blockIdx.z == 0) {  // constants: ahead of the dependency wait
        bias = __ldg(reinterpret_cast<const float4*>(a.conv_b + c));
#pragma unroll
        for (int j = 0; j < TAPS; ++j) w[j] = __ldg(reinterpret_cast<const float4*>(a.conv_w + (size_t)j * a.inner_rows + c));
    }
    pdl_wait();
    if (!ok && tid == 0) atomicOr(&a.st->status, kStatusBadPos);
    if (!ok || !in) return;
    if (blockIdx.z == 1) {
        float4 v[kConvTokens];
        prefill_sums(a.part, n_rows, a.splits, a.n_tokens, t0, a.inner_rows + c, v);
#pragma unroll
        for (int i = 0; i < kConvTokens; ++i)
            if (t0 + i < a.n_tokens) *reinterpret_cast<float4*>(a.z + (size_t)(t0 + i) * a.x_pitch + c) = silu4(v[i]);
        return;
    }
    // Input i of the thread is that of token t0 - slots + i: a product, from the ring, or zero before the first position.
    auto earlier = [&](int i, const float4& v) -> float4 {
        const int pos = a.start_pos + t0 - slots + i;
        if (t0 - slots + i >= 0) return v;
        return pos < 0 ? zero : __ldcg(reinterpret_cast<const float4*>(a.ring + (size_t)(pos % slots) * a.inner_rows + c));
    };
    auto keep = [&](int i, const float4& v) {
        const int t = t0 - slots + i;
        if (t >= t0 && t >= a.n_tokens - slots && t < a.n_tokens)
            *reinterpret_cast<float4*>(a.tail + (size_t)((a.start_pos + t) % slots) * a.inner_rows + c) = v;
    };
    auto put = [&](int i, const float4& sum) {
        const int t = t0 + i;
        if (t >= a.n_tokens) return;
        const float4 v = silu4(sum);
        *reinterpret_cast<float4*>(a.x + (size_t)t * a.x_pitch + c) = v;
        const float x[4] = {v.x, v.y, v.z, v.w};
        __align__(8) __nv_bfloat16 hi[4], lo[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) split_pair(x[k], hi[k], lo[k]);
        *reinterpret_cast<uint2*>(a.planes + (size_t)t * a.x_pitch + c) = *reinterpret_cast<const uint2*>(hi);
        *reinterpret_cast<uint2*>(a.planes + (size_t)(kPrefillTokens + t) * a.x_pitch + c) = *reinterpret_cast<const uint2*>(lo);
    };
    if constexpr (TAPS > 0) {
        constexpr int N = kConvTokens + TAPS - 1;
        float4 v[N];
        prefill_sums(a.part, n_rows, a.splits, a.n_tokens, t0 - slots, c, v);
        if constexpr (TAPS > 1) {
            if (t0 < slots)
#pragma unroll
                for (int i = 0; i < TAPS - 1; ++i) v[i] = earlier(i, v[i]);
            if (t0 + kConvTokens > a.n_tokens - slots)
#pragma unroll
                for (int i = 0; i < N; ++i) keep(i, v[i]);
        }
#pragma unroll
        for (int i = 0; i < kConvTokens; ++i) {
            float4 s = bias;
#pragma unroll
            for (int j = 0; j < TAPS; ++j) s = fma4(w[j], v[i + j], s);
            put(i, s);
        }
    } else {
        for (int i = 0; i < kConvTokens + slots; ++i) {
            float4 v[1];
            prefill_sums(a.part, n_rows, a.splits, a.n_tokens, t0 - slots + i, c, v);
            v[0] = earlier(i, v[0]);
            if (slots > 0) keep(i, v[0]);
            cv_in[i * kConvThreads + tid] = v[0];
        }
        for (int i = 0; i < kConvTokens; ++i) {
            float4 s = bias;
            for (int j = 0; j <= slots; ++j)
                s = fma4(__ldg(reinterpret_cast<const float4*>(a.conv_w + (size_t)j * a.inner_rows + c)), cv_in[(i + j) * kConvThreads + tid], s);
            put(i, s);
        }
    }
}

// dt | B | C rows after their GEMM, whose row tiles are few and whose K is therefore cut into up to kLowMaxSplits ranges:
// partial sums added in range order (in kLowGroups groups), sections padded with zeros to dt_pitch and state_pitch.
// grid: (tokens, ceil(row / kLowColumns))
constexpr int kLowMaxSplits = 32, kLowColumns = 64, kLowGroups = 4, kLowThreads = kLowColumns * kLowGroups;
// floats per row, an odd number of 16-byte pieces (rows on different banks of shared memory)
__host__ __device__ inline int mamba_low_pitch(int dt_pitch, int state_pitch) {
    const int n = dt_pitch + 2 * state_pitch;
    return (n / 4) % 2 ? n : n + 4;
}
static __global__ void __launch_bounds__(kLowThreads) mamba_low_kernel(const MambaScanArgs a, const float* part, int splits, float* out) {
    __shared__ float group_sum[kLowGroups][kLowColumns];
    pdl_launch_dependents();
    const int t = blockIdx.x, tid = threadIdx.x, col = tid % kLowColumns, group = tid / kLowColumns, i = (int)blockIdx.y * kLowColumns + col;
    const int src = mamba_low_source(a, i);  // -1: padding
    constexpr int N = kLowMaxSplits / kLowGroups;
    const int per = (splits + kLowGroups - 1) / kLowGroups, s0 = group * per, n = min(per, splits - s0);
    pdl_wait();
    const float* p = part + ((size_t)s0 * kPrefillTokens + t) * a.low_rows + max(src, 0);
    float v[N], sum = 0.f;
#pragma unroll
    for (int s = 0; s < N; ++s) v[s] = s < n ? __ldcg(p + (size_t)s * kPrefillTokens * a.low_rows) : 0.f;
#pragma unroll
    for (int s = 0; s < N; ++s) sum += v[s];
    group_sum[group][col] = sum;
    __syncthreads();
    if (group != 0 || i >= a.dt_pitch + 2 * a.state_pitch) return;
    sum = 0.f;
#pragma unroll
    for (int g = 0; g < kLowGroups; ++g) sum += group_sum[g][col];
    out[(size_t)t * mamba_low_pitch(a.dt_pitch, a.state_pitch) + i] = src >= 0 ? sum : 0.f;
}

// The recurrence over a prompt block.  A CTA owns kScanThreads / L channels and walks the block in tiles of tile_tokens:
// dt | B | C rows, x and z to shared memory, dt = softplus(W_dt . + bias) for all tokens and channels of the tile, then
// four tokens at a time with the state in registers.
constexpr int kScanThreads = 128;
template <int L>
constexpr int kScanChannels = kScanThreads / L;
template <int L>
__host__ __device__ inline int mamba_scan_smem(int dt_pitch, int state_pitch, int tile_tokens) {
    return (tile_tokens * (mamba_low_pitch(dt_pitch, state_pitch) + 3 * kScanChannels<L>) + kScanChannels<L> * (dt_pitch + 4)) * 4;
}
// Sums over the L lanes of a channel of four values each (one per token); lane ln gets that of token scan_token(ln).
__device__ __forceinline__ int scan_token(int ln) { return ((ln & 1) << 1) | ((ln >> 1) & 1); }
template <int L>
__device__ __forceinline__ float lane_group_sum4(const float (&y)[4], int ln) {
    static_assert(L >= 4, "four tokens to four lanes");
    const bool b0 = ln & 1, b1 = ln & 2;
    float p = b0 ? y[2] : y[0], q = b0 ? y[3] : y[1];
    p += __shfl_xor_sync(0xffffffffu, b0 ? y[0] : y[2], 1);
    q += __shfl_xor_sync(0xffffffffu, b0 ? y[1] : y[3], 1);
    float r = b1 ? q : p;
    r += __shfl_xor_sync(0xffffffffu, b1 ? p : q, 2);
#pragma unroll
    for (int o = 4; o < L; o <<= 1) r += __shfl_xor_sync(0xffffffffu, r, o);
    return r;
}
template <int L, int NS>
static __global__ void __launch_bounds__(kScanThreads) mamba_scan_kernel(const MambaScanArgs a) {
    constexpr int CH = kScanChannels<L>;
    constexpr int TX = CH < 8 ? CH : 8, CPT = CH / TX, TY = kScanThreads / TX, TPT = 4;  // dt product: channels x tokens per thread
    extern __shared__ __align__(16) float sm_scan[];
    const int LP = mamba_low_pitch(a.dt_pitch, a.state_pitch), WP = a.dt_pitch + 4;
    float* low = sm_scan;                       // [tile_tokens][LP]
    float* wd = low + a.tile_tokens * LP;       // [CH][WP]
    float* xs = wd + CH * WP;                   // [tile_tokens][CH]: x, then y
    float* zs = xs + a.tile_tokens * CH;        // [tile_tokens][CH]
    float* dts = zs + a.tile_tokens * CH;       // [tile_tokens][CH]
    const int tid = threadIdx.x, ln = tid % L, cl = tid / L, c0 = blockIdx.x * CH, c = c0 + cl;
    const bool in = c < a.inner;
    constexpr int pieces = L * NS;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    const float4* A4 = reinterpret_cast<const float4*>(a.A) + (size_t)(in ? c : 0) * pieces + ln;
    float4* S4 = reinterpret_cast<float4*>(a.S) + (size_t)(in ? c : 0) * pieces + ln;
    pdl_launch_dependents();
    // weights: ahead of the dependency wait
    for (int i = tid; i < CH * (a.dt_pitch / 8); i += kScanThreads) {
        const int r = i / (a.dt_pitch / 8), v = i - r * (a.dt_pitch / 8);
        uint4 u = make_uint4(0, 0, 0, 0);
        if (c0 + r < a.inner) u = ldg_stream_u4(reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(a.w_dt) + (size_t)(c0 + r) * a.dt_pitch) + v);
        float* d = wd + r * WP + v * 8;
        const float2 f0 = bf162_bits_to_float2(u.x), f1 = bf162_bits_to_float2(u.y), f2 = bf162_bits_to_float2(u.z), f3 = bf162_bits_to_float2(u.w);
        *reinterpret_cast<float4*>(d) = make_float4(f0.x, f0.y, f1.x, f1.y);
        *reinterpret_cast<float4*>(d + 4) = make_float4(f2.x, f2.y, f3.x, f3.y);
    }
    ScanPiece A[NS], S[NS];
#pragma unroll
    for (int i = 0; i < NS; ++i) A[i] = scan_piece(__ldg(A4 + i * L));
    const float D = in ? __ldg(a.D + c) : 0.f;
    const int tx = tid % TX, ty = tid / TX;
    float bias[CPT];
#pragma unroll
    for (int j = 0; j < CPT; ++j) bias[j] = c0 + tx + j * TX < a.inner ? __ldg(a.dt_b + c0 + tx + j * TX) : 0.f;
    pdl_wait();
    if (a.start_pos < 0 || a.start_pos + a.n_tokens > a.seq_len) return;
    for (int t0 = 0; t0 < a.n_tokens; t0 += a.tile_tokens) {
        const int nt = min(a.tile_tokens, a.n_tokens - t0);
        if (t0 > 0) __syncthreads();
        for (int i = tid; i < nt * (LP / 4); i += kScanThreads) cp_async_16(low + 4 * i, a.low + (size_t)t0 * LP + 4 * i, true);
        for (int i = tid; i < nt * (CH / 4); i += kScanThreads) {  // x_pitch is a multiple of 64: no row ends inside a piece
            const int t = i / (CH / 4), k = 4 * (i - t * (CH / 4));
            const size_t at = (size_t)(t0 + t) * a.x_pitch + c0 + k;
            const bool have = c0 + k < a.x_pitch;
            cp_async_16(xs + t * CH + k, a.x + (have ? at : 0), have);
            cp_async_16(zs + t * CH + k, a.z + (have ? at : 0), have);
        }
        cp_async_commit();
        if (t0 == 0) {
#pragma unroll
            for (int i = 0; i < NS; ++i) S[i] = scan_piece(a.start_pos > 0 ? __ldcg(S4 + i * L) : zero);
            // the convolution inputs that the next portion needs
            if (a.taps > 1) {
                const int slots = a.taps - 1, keep = min(slots, a.n_tokens);
                for (int i = tid; i < keep * CH; i += kScanThreads) {
                    const int k = i / CH, ch = c0 + i - k * CH;
                    const size_t at = (size_t)((a.start_pos + a.n_tokens - 1 - k) % slots) * a.ring_pitch + ch;
                    if (ch < a.inner) a.ring[at] = __ldcg(a.tail + at);
                }
            }
        }
        cp_async_wait<0>();
        __syncthreads();
        for (int tb = 0; tb < nt; tb += TPT * TY) {
            f32x2 acc[TPT][CPT];
#pragma unroll
            for (int i = 0; i < TPT; ++i)
#pragma unroll
                for (int j = 0; j < CPT; ++j) acc[i][j] = both(0.f);
            int at[TPT];
#pragma unroll
            for (int i = 0; i < TPT; ++i) at[i] = min(tb + ty + i * TY, nt - 1) * LP;  // beyond the tile: not used
#pragma unroll 2
            for (int k = 0; k < a.dt_pitch; k += 4) {
                ScanPiece l[TPT], w[CPT];
#pragma unroll
                for (int i = 0; i < TPT; ++i) l[i] = scan_piece(*reinterpret_cast<const float4*>(low + at[i] + k));
#pragma unroll
                for (int j = 0; j < CPT; ++j) w[j] = scan_piece(*reinterpret_cast<const float4*>(wd + (tx + j * TX) * WP + k));
#pragma unroll
                for (int i = 0; i < TPT; ++i)
#pragma unroll
                    for (int j = 0; j < CPT; ++j) acc[i][j] = fma2(l[i].hi, w[j].hi, fma2(l[i].lo, w[j].lo, acc[i][j]));
            }
#pragma unroll
            for (int i = 0; i < TPT; ++i) {
                const int t = tb + ty + i * TY;
#pragma unroll
                for (int j = 0; j < CPT; ++j)  // a step of size 0 leaves the state alone: what fills up the last four tokens
                    if (t < a.tile_tokens) dts[t * CH + tx + j * TX] = t < nt ? softplus_f(pair_sum(acc[i][j]) + bias[j]) : 0.f;
            }
        }
        __syncthreads();
        for (int t = 0; t < nt; t += 4) {
            float y[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const int tk = min(t + k, nt - 1);
                const float dt = dts[(t + k) * CH + cl], dx = dt * xs[tk * CH + cl];
                const float4* B = reinterpret_cast<const float4*>(low + tk * LP + a.dt_pitch);
                f32x2 y2 = both(0.f);
#pragma unroll
                for (int i = 0; i < NS; ++i)
                    mamba_update(S[i], A[i], scan_piece(B[ln + i * L]), scan_piece(B[pieces + ln + i * L]), both(dt), both(dx), y2);
                y[k] = pair_sum(y2);
            }
            const float sum = lane_group_sum4<L>(y, ln);
            const int mine = t + scan_token(ln);
            __syncwarp();  // the channel's lanes have read x
            if (ln < 4 && mine < nt) xs[mine * CH + cl] = fmaf(D, xs[mine * CH + cl], sum);
        }
        __syncthreads();
        for (int i = tid; i < nt * (CH / 2); i += kScanThreads) {
            const int t = i / (CH / 2), ch = 2 * (i - t * (CH / 2));
            if (c0 + ch >= a.inner) continue;
            __align__(4) __nv_bfloat16 hi[2], lo[2];
            split_pair(xs[t * CH + ch] * zs[t * CH + ch], hi[0], lo[0]);
            split_pair(c0 + ch + 1 < a.inner ? xs[t * CH + ch + 1] * zs[t * CH + ch + 1] : 0.f, hi[1], lo[1]);
            __nv_bfloat16* d = a.planes + (size_t)(t0 + t) * a.plane_row + c0 + ch;
            *reinterpret_cast<uint32_t*>(d) = *reinterpret_cast<const uint32_t*>(hi);
            *reinterpret_cast<uint32_t*>(d + (size_t)kPrefillTokens * a.plane_row) = *reinterpret_cast<const uint32_t*>(lo);
        }
    }
    if (!in) return;
#pragma unroll
    for (int i = 0; i < NS; ++i) S4[i * L] = scan_float4(S[i]);
}

}  // namespace lpp
