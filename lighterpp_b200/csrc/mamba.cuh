// Selective-scan layers (Mamba): a recurrence per channel whose step size, input and output vectors depend on the token.
//
//   x | z  = W_in h                     x: causal convolution over the last `taps` tokens, silu      z: silu
//   dt | B | C = W_x x                  dt: softplus(W_dt dt + bias), one per channel
//   S[c,n] <- exp(dt_c A[c,n]) S[c,n] + dt_c x_c B_n        y_c = sum_n S[c,n] C_n + D_c x_c        out = W_o (y * z)
//
// (Albert Gu, Tri Dao: Mamba: Linear-Time Sequence Modeling with Selective State Spaces.)  A decode step of a layer has four
// kernels: the input GEMV (its epilogue is the convolution), the GEMV of W_x, the scan (which also multiplies with W_dt: a
// channel's row of it belongs to the lanes that own the channel's state) and the output GEMV with the residual.  A prompt
// block has the same products as GEMMs, with the convolution and the scan as kernels of their own (prefill_mixers.cuh); the
// scan walks the block's tokens with the state in registers.
//
// What a sequence leaves behind: S [inner][state] and the last taps - 1 convolution inputs, all FP32.  The input of position
// p lies in slot p % (taps - 1), so nothing moves when a token is added and positions before 0 are never read: a new
// sequence needs no clearing (the state of a sequence at position 0 counts as zero).
#pragma once
#include "common.cuh"

namespace lpp {

// ---- input projection of a step: rows  x [inner_rows] | z [inner_rows]

struct MambaInArgs {
    int inner, inner_rows;  // channels, rounded up to even
    int taps;
    int early;              // weights and state may be read before the dependency wait (and so may the position)
    const float* conv_w;    // [taps][inner_rows]
    const float* conv_b;    // [inner_rows]
    float* ring;            // [taps - 1][inner_rows]
    float* x;               // [inner], convolved
    float* z;               // [inner], through the silu
};

// The convolution of row `row` without the current token, and the current token's tap.
__device__ __forceinline__ RowPrep mamba_in_prep(const MambaInArgs& m, int pos, int row) {
    RowPrep p;
    if (row >= m.inner) return p;
    const int slots = m.taps - 1;
    p.x = __ldg(m.conv_b + row);
    p.y = __ldg(m.conv_w + (size_t)slots * m.inner_rows + row);
#pragma unroll 4
    for (int back = slots; back >= 1; --back)
        if (pos >= back)
            p.x = fmaf(__ldg(m.conv_w + (size_t)(slots - back) * m.inner_rows + row),
                       __ldcg(m.ring + (size_t)((pos - back) % slots) * m.inner_rows + row), p.x);
    return p;
}
__device__ __forceinline__ void mamba_in_row(const MambaInArgs& m, int pos, int row, float v, const RowPrep& p) {
    const bool is_x = row < m.inner_rows;
    const int c = is_x ? row : row - m.inner_rows;
    if (c >= m.inner) return;
    if (!is_x) {
        m.z[c] = silu_f(v);
        return;
    }
    if (m.taps > 1) m.ring[(size_t)(pos % (m.taps - 1)) * m.inner_rows + c] = v;
    m.x[c] = silu_f(fmaf(p.y, v, p.x));
}

// ---- the recurrence.  A channel's state belongs to L neighbouring lanes, each of which holds NS pieces of four elements
// (piece q of the channel to lane q % L).

struct MambaScanArgs {
    int inner, state, dt_rank;
    int state_pitch, dt_pitch;  // elements per channel of S and A (multiple of 4), of w_dt (multiple of 8)
    int low_rows;               // row of `low`: dt | B | C, even
    const float* low;           // step: [low_rows]; prompt block: [kPrefillTokens][mamba_low_pitch], padded
    const void* w_dt;           // [inner][dt_pitch], weight type
    const float *dt_b, *A, *D;  // [inner], [inner][state_pitch] (negative), [inner]
    float* S;                   // [inner][state_pitch]
    const float *x, *z;         // step: [inner]; prompt block: [kPrefillTokens][x_pitch]
    float* out;                 // step: [inner]
    StepState* st;
    int seq_len;
    int early;                  // step: weights and state may be read before the dependency wait
    // prompt block
    int n_tokens, start_pos, x_pitch;
    int tile_tokens;            // tokens whose rows fit shared memory together (a multiple of 4)
    __nv_bfloat16* planes;      // [2 planes][kPrefillTokens][plane_row]
    int plane_row;
    const float* tail;          // convolution inputs of the block's last tokens, laid out like the ring
    float* ring;
    int taps, ring_pitch;
};

// exp(x) - 1 for x <= 0.  A channel that forgets slowly multiplies its state with a factor just below 1 thousands of times,
// and always with much the same one: the rounding of the factor itself to 32 bits (2^-25 of it, the same way every time)
// would add up, so the state is updated with its difference from 1.  Taylor series where it cancels (the first term left
// out is below 2e-8 of the sum).
__device__ __forceinline__ float decay_m1(float x) {
    float p = fmaf(x, 1.f / 40320.f, 1.f / 5040.f);
    p = fmaf(x, p, 1.f / 720.f);
    p = fmaf(x, p, 1.f / 120.f);
    p = fmaf(x, p, 1.f / 24.f);
    p = fmaf(x, p, 1.f / 6.f);
    p = fmaf(x, p, 0.5f);
    p = fmaf(x * x, p, x);
    return x > -0.5f ? p : __expf(x) - 1.f;
}
// S <- exp(dt A) S + dx B
__device__ __forceinline__ void state_update(float& S, float A, float B, float dt, float dx) {
    S = fmaf(decay_m1(dt * A), S, fmaf(dx, B, S));
}
// The same for four elements; returns their share of S . C
__device__ __forceinline__ float mamba_update(float4& S, const float4& A, const float4& B, const float4& C, float dt, float dx) {
    state_update(S.x, A.x, B.x, dt, dx);
    state_update(S.y, A.y, B.y, dt, dx);
    state_update(S.z, A.z, B.z, dt, dx);
    state_update(S.w, A.w, B.w, dt, dx);
    return fmaf(S.x, C.x, fmaf(S.y, C.y, fmaf(S.z, C.z, S.w * C.w)));
}
template <int L>
__device__ __forceinline__ float lane_group_sum(float v) {
#pragma unroll
    for (int o = L / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
// Element i of a token's dt | B | C row with dt padded to dt_pitch, B and C to state_pitch, with zeros.
__device__ __forceinline__ float mamba_low(const MambaScanArgs& a, const float* src, int i) {
    int n = a.dt_rank, from = 0;
    if (i >= a.dt_pitch) {
        i -= a.dt_pitch;
        n = a.state;
        from = a.dt_rank;
        if (i >= a.state_pitch) i -= a.state_pitch, from += a.state;
    }
    return i < n ? __ldcg(src + from + i) : 0.f;
}

// One token.  grid: ceil(inner / (kScanStepThreads / L)); shared memory: dt_pitch + 2 state_pitch floats
constexpr int kScanStepThreads = 64;
template <typename WT, int L, int NS>
static __global__ void __launch_bounds__(kScanStepThreads) mamba_step_kernel(const MambaScanArgs a) {
    extern __shared__ __align__(16) float sc_low[];
    constexpr int kVec = 16 / sizeof(WT), kAhead = 4;  // weights per 16-byte load; loads of W_dt ahead of the wait
    const int tid = threadIdx.x, ln = tid % L, c = blockIdx.x * (kScanStepThreads / L) + tid / L;
    const bool in = c < a.inner;
    pdl_launch_dependents();
    if (!a.early) pdl_wait();
    const int pos = a.st->pos;
    const bool ok = pos >= 0 && pos < a.seq_len;
    const int pieces = a.state_pitch / 4, vecs = a.dt_pitch / kVec;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    float4 A[NS], S[NS];
#pragma unroll
    for (int i = 0; i < NS; ++i) {
        const int q = ln + i * L;
        const bool have = in && q < pieces;
        A[i] = have ? __ldg(reinterpret_cast<const float4*>(a.A + (size_t)c * a.state_pitch) + q) : zero;
        S[i] = have && pos > 0 ? __ldcg(reinterpret_cast<const float4*>(a.S + (size_t)c * a.state_pitch) + q) : zero;
    }
    const uint4* w = reinterpret_cast<const uint4*>(reinterpret_cast<const WT*>(a.w_dt) + (size_t)(in ? c : 0) * a.dt_pitch);
    uint4 wv[kAhead];
#pragma unroll
    for (int i = 0; i < kAhead; ++i)
        if (ln + i * L < vecs) wv[i] = ldg_stream_u4(w + ln + i * L);
    const float bias = in ? __ldg(a.dt_b + c) : 0.f, D = in ? __ldg(a.D + c) : 0.f;
    pdl_wait();
    const float x = in ? __ldcg(a.x + c) : 0.f, z = in ? __ldcg(a.z + c) : 0.f;
    for (int i = tid; i < a.dt_pitch + 2 * a.state_pitch; i += kScanStepThreads) sc_low[i] = mamba_low(a, a.low, i);
    __syncthreads();
    float dot = 0.f;
    auto mul = [&](const uint4& u, int v) {
        const float* d = sc_low + v * kVec;
        const uint32_t q[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            if constexpr (sizeof(WT) == 2) {
                const float2 f = unpack2<WT>(q[i]);
                dot = fmaf(f.x, d[2 * i], dot);
                dot = fmaf(f.y, d[2 * i + 1], dot);
            } else {
                dot = fmaf(__uint_as_float(q[i]), d[i], dot);
            }
        }
    };
#pragma unroll
    for (int i = 0; i < kAhead; ++i)
        if (ln + i * L < vecs) mul(wv[i], ln + i * L);
    for (int v = ln + kAhead * L; v < vecs; v += L) mul(ldg_stream_u4(w + v), v);
    const float dt = softplus_f(lane_group_sum<L>(dot) + bias);
    const float4* B = reinterpret_cast<const float4*>(sc_low + a.dt_pitch);
    const float4* C = B + pieces;
    float y = 0.f;
#pragma unroll
    for (int i = 0; i < NS; ++i) {
        const int q = ln + i * L;
        if (q < pieces) y += mamba_update(S[i], A[i], B[q], C[q], dt, dt * x);
    }
    y = lane_group_sum<L>(y);
    if (!in || !ok) return;
#pragma unroll
    for (int i = 0; i < NS; ++i)
        if (ln + i * L < pieces) *(reinterpret_cast<float4*>(a.S + (size_t)c * a.state_pitch) + ln + i * L) = S[i];
    if (ln == 0) a.out[c] = fmaf(D, x, y) * z;
}

}  // namespace lpp
