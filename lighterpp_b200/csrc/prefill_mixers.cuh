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
// One row alone.
__device__ __forceinline__ float prefill_sum1(const float* part, int n_rows, int splits, int t, int row) {
    float p[kPfMaxSplits], v = 0.f;
#pragma unroll
    for (int s = 0; s < kPfMaxSplits; ++s)
        if (s < splits) p[s] = part[((size_t)s * kPrefillTokens + t) * n_rows + row];
#pragma unroll
    for (int s = 0; s < kPfMaxSplits; ++s)
        if (s < splits) v += p[s];
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
// copies them to the ring once every CTA of this launch has read it.
// grid: (ceil(inner / 128), ceil(tokens / 8), 2: x, z); shared memory (x): (8 + taps - 1) * 128 floats
constexpr int kConvChannels = 128, kConvTokens = 8;
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
static __global__ void __launch_bounds__(kConvChannels) mamba_conv_kernel(const MambaConvArgs a) {
    extern __shared__ float cv_in[];  // [kConvTokens + taps - 1][kConvChannels]; a thread reads back only what it wrote
    pdl_launch_dependents();
    const int tid = threadIdx.x, c = blockIdx.x * kConvChannels + tid;
    const int t0 = blockIdx.y * kConvTokens, t1 = min(t0 + kConvTokens, a.n_tokens);
    const int n_rows = 2 * a.inner_rows, slots = a.taps - 1;
    pdl_wait();
    if (a.start_pos < 0 || a.start_pos + a.n_tokens > a.seq_len) {
        if (tid == 0) atomicOr(&a.st->status, kStatusBadPos);
        return;
    }
    if (c >= a.inner) return;
    if (blockIdx.z == 1) {
#pragma unroll 4
        for (int t = t0; t < t1; ++t) a.z[(size_t)t * a.x_pitch + c] = silu_f(prefill_sum1(a.part, n_rows, a.splits, t, a.inner_rows + c));
        return;
    }
#pragma unroll 4
    for (int t = t0 - slots; t < t1; ++t) {
        float v = 0.f;
        if (t >= 0)
            v = prefill_sum1(a.part, n_rows, a.splits, t, c);
        else if (a.start_pos + t >= 0)
            v = __ldcg(a.ring + (size_t)((a.start_pos + t) % slots) * a.inner_rows + c);
        cv_in[(t - t0 + slots) * kConvChannels + tid] = v;
        if (t >= t0 && t >= a.n_tokens - slots) a.tail[(size_t)((a.start_pos + t) % slots) * a.inner_rows + c] = v;
    }
    const float bias = __ldg(a.conv_b + c);
    for (int t = t0; t < t1; ++t) {
        float v = bias;
#pragma unroll 4
        for (int j = 0; j < a.taps; ++j) v = fmaf(__ldg(a.conv_w + (size_t)j * a.inner_rows + c), cv_in[(t - t0 + j) * kConvChannels + tid], v);
        v = silu_f(v);
        a.x[(size_t)t * a.x_pitch + c] = v;
        __nv_bfloat16 hi, lo;
        split_pair(v, hi, lo);
        a.planes[(size_t)t * a.x_pitch + c] = hi;
        a.planes[(size_t)(kPrefillTokens + t) * a.x_pitch + c] = lo;
    }
}

// The recurrence over a prompt block.  A CTA owns kScanThreads / L channels and walks the block in tiles of tile_tokens:
// dt | B | C rows to shared memory (partial sums of the W_x GEMM added in range order), dt = softplus(W_dt . + bias) for all
// tokens and channels of the tile, then token by token with the state in registers.
constexpr int kScanThreads = 128;
template <int L>
constexpr int kScanChannels = kScanThreads / L;
// floats per token row in shared memory, an odd number of 16-byte pieces (rows on different banks)
__host__ __device__ inline int mamba_low_pitch(int dt_pitch, int state_pitch) {
    const int n = dt_pitch + 2 * state_pitch;
    return (n / 4) % 2 ? n : n + 4;
}
template <int L>
__host__ __device__ inline int mamba_scan_smem(int dt_pitch, int state_pitch, int tile_tokens) {
    return (tile_tokens * (mamba_low_pitch(dt_pitch, state_pitch) + 2 * kScanChannels<L>) + kScanChannels<L> * (dt_pitch + 4)) * 4;
}
template <int L, int NS>
static __global__ void __launch_bounds__(kScanThreads) mamba_scan_kernel(const MambaScanArgs a) {
    constexpr int CH = kScanChannels<L>;
    constexpr int TX = CH < 8 ? CH : 8, CPT = CH / TX, TY = kScanThreads / TX, TPT = 4;  // dt product: channels x tokens per thread
    extern __shared__ __align__(16) float sm_scan[];
    const int LP = mamba_low_pitch(a.dt_pitch, a.state_pitch), WP = a.dt_pitch + 4;
    float* low = sm_scan;                       // [tile_tokens][LP]
    float* wd = low + a.tile_tokens * LP;       // [CH][WP]
    float* dts = wd + CH * WP;                  // [tile_tokens][CH]
    float* xs = dts + a.tile_tokens * CH;       // [tile_tokens][CH]: x, then y
    const int tid = threadIdx.x, ln = tid % L, cl = tid / L, c0 = blockIdx.x * CH, c = c0 + cl;
    const bool in = c < a.inner;
    const int pieces = a.state_pitch / 4;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
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
    float4 A[NS], S[NS];
#pragma unroll
    for (int i = 0; i < NS; ++i) A[i] = in && ln + i * L < pieces ? __ldg(reinterpret_cast<const float4*>(a.A + (size_t)c * a.state_pitch) + ln + i * L) : zero;
    const float D = in ? __ldg(a.D + c) : 0.f;
    const int tx = tid % TX, ty = tid / TX;
    float bias[CPT];
#pragma unroll
    for (int j = 0; j < CPT; ++j) bias[j] = c0 + tx + j * TX < a.inner ? __ldg(a.dt_b + c0 + tx + j * TX) : 0.f;
    pdl_wait();
    if (a.start_pos < 0 || a.start_pos + a.n_tokens > a.seq_len) return;
#pragma unroll
    for (int i = 0; i < NS; ++i)
        S[i] = in && a.start_pos > 0 && ln + i * L < pieces ? __ldcg(reinterpret_cast<const float4*>(a.S + (size_t)c * a.state_pitch) + ln + i * L) : zero;
    // the convolution inputs that the next portion needs
    if (a.taps > 1) {
        const int slots = a.taps - 1, keep = min(slots, a.n_tokens);
        for (int i = tid; i < keep * CH; i += kScanThreads) {
            const int k = i / CH, ch = c0 + i - k * CH;
            const size_t at = (size_t)((a.start_pos + a.n_tokens - 1 - k) % slots) * a.ring_pitch + ch;
            if (ch < a.inner) a.ring[at] = __ldcg(a.tail + at);
        }
    }
    for (int t0 = 0; t0 < a.n_tokens; t0 += a.tile_tokens) {
        const int nt = min(a.tile_tokens, a.n_tokens - t0);
        if (t0 > 0) __syncthreads();
        // dt | B | C rows
        const int n_low = a.dt_pitch + 2 * a.state_pitch;
        for (int i = tid; i < nt * n_low; i += kScanThreads) {
            const int t = i / n_low, k = i - t * n_low;
            float v[kPfMaxSplits], sum = 0.f;
#pragma unroll
            for (int s = 0; s < kPfMaxSplits; ++s)
                if (s < a.splits) v[s] = mamba_low(a, a.low + ((size_t)s * kPrefillTokens + t0 + t) * a.low_rows, k);
#pragma unroll
            for (int s = 0; s < kPfMaxSplits; ++s)
                if (s < a.splits) sum += v[s];
            low[t * LP + k] = sum;
        }
        for (int i = tid; i < nt * CH; i += kScanThreads) {
            const int t = i / CH, ch = i - t * CH;
            xs[i] = c0 + ch < a.inner ? __ldcg(a.x + (size_t)(t0 + t) * a.x_pitch + c0 + ch) : 0.f;
        }
        __syncthreads();
        for (int tb = 0; tb < nt; tb += TPT * TY) {
            float acc[TPT][CPT];
#pragma unroll
            for (int i = 0; i < TPT; ++i)
#pragma unroll
                for (int j = 0; j < CPT; ++j) acc[i][j] = 0.f;
            int at[TPT];
#pragma unroll
            for (int i = 0; i < TPT; ++i) at[i] = min(tb + ty + i * TY, nt - 1) * LP;  // beyond the tile: not stored
            for (int k = 0; k < a.dt_pitch; k += 4) {
                float4 l[TPT], w[CPT];
#pragma unroll
                for (int i = 0; i < TPT; ++i) l[i] = *reinterpret_cast<const float4*>(low + at[i] + k);
#pragma unroll
                for (int j = 0; j < CPT; ++j) w[j] = *reinterpret_cast<const float4*>(wd + (tx + j * TX) * WP + k);
#pragma unroll
                for (int i = 0; i < TPT; ++i)
#pragma unroll
                    for (int j = 0; j < CPT; ++j)
                        acc[i][j] = fmaf(l[i].x, w[j].x, fmaf(l[i].y, w[j].y, fmaf(l[i].z, w[j].z, fmaf(l[i].w, w[j].w, acc[i][j]))));
            }
#pragma unroll
            for (int i = 0; i < TPT; ++i) {
                const int t = tb + ty + i * TY;
#pragma unroll
                for (int j = 0; j < CPT; ++j)
                    if (t < nt) dts[t * CH + tx + j * TX] = softplus_f(acc[i][j] + bias[j]);
            }
        }
        __syncthreads();
#pragma unroll 4
        for (int t = 0; t < nt; ++t) {
            const float dt = dts[t * CH + cl], x = xs[t * CH + cl];
            const float4* B = reinterpret_cast<const float4*>(low + t * LP + a.dt_pitch);
            float y = 0.f;
#pragma unroll
            for (int i = 0; i < NS; ++i) {
                const int q = ln + i * L;
                if (q < pieces) y += mamba_update(S[i], A[i], B[q], B[pieces + q], dt, dt * x);
            }
            y = lane_group_sum<L>(y);
            __syncwarp();  // the channel's lanes have read x
            if (ln == 0) xs[t * CH + cl] = fmaf(D, x, y);
        }
        __syncthreads();
        for (int i = tid; i < nt * CH; i += kScanThreads) {
            const int t = i / CH, ch = i - t * CH;
            if (c0 + ch >= a.inner) continue;
            const float v = xs[i] * __ldcg(a.z + (size_t)(t0 + t) * a.x_pitch + c0 + ch);
            __nv_bfloat16 hi, lo;
            split_pair(v, hi, lo);
            __nv_bfloat16* d = a.planes + (size_t)(t0 + t) * a.plane_row + c0 + ch;
            d[0] = hi;
            d[(size_t)kPrefillTokens * a.plane_row] = lo;
        }
    }
    if (!in) return;
#pragma unroll
    for (int i = 0; i < NS; ++i)
        if (ln + i * L < pieces) *(reinterpret_cast<float4*>(a.S + (size_t)c * a.state_pitch) + ln + i * L) = S[i];
}

}  // namespace lpp
