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
    int inner, inner_rows;  // channels, rounded up to a multiple of 4
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
// (piece q of the channel to lane q % L).  In memory a channel has 4 L NS elements, the ones beyond its state zero: they stay
// zero, because the same holds for A, B and C.

struct MambaScanArgs {
    int inner, state, dt_rank;
    int state_pitch, dt_pitch;  // elements per channel of S and A (4 L NS), of w_dt (multiple of 8)
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

// Pairs of floats in one 64-bit register: sm_100 multiplies and adds both with one instruction.
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack_f2(float lo, float hi) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ float2 unpack_f2(f32x2 v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
    f32x2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
__device__ __forceinline__ f32x2 both(float v) { return pack_f2(v, v); }
__device__ __forceinline__ float exp2_approx(float x) {
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
    return r;
}

// exp(x) - 1 for x <= 0.  A channel that forgets slowly multiplies its state with a factor just below 1 thousands of times,
// and always with much the same one: the rounding of the factor itself to 32 bits (2^-25 of it, the same way every time)
// would add up, so the state is updated with its difference from 1.  Taylor series where it cancels (the first term left
// out is below 5e-8 of the sum).
__device__ __forceinline__ f32x2 decay_m1(f32x2 x) {
    f32x2 p = fma2(x, both(1.f / 720.f), both(1.f / 120.f));
    p = fma2(x, p, both(1.f / 24.f));
    p = fma2(x, p, both(1.f / 6.f));
    p = fma2(x, p, both(0.5f));
    p = fma2(mul2(x, x), p, x);
    const float2 v = unpack_f2(x), series = unpack_f2(p), t = unpack_f2(mul2(x, both(1.4426950408889634f)));
    return pack_f2(v.x > -0.25f ? series.x : exp2_approx(t.x) - 1.f, v.y > -0.25f ? series.y : exp2_approx(t.y) - 1.f);
}
// Four elements of a channel, as two pairs.
struct ScanPiece {
    f32x2 lo, hi;
};
__device__ __forceinline__ ScanPiece scan_piece(const float4& v) { return {pack_f2(v.x, v.y), pack_f2(v.z, v.w)}; }
__device__ __forceinline__ float4 scan_float4(const ScanPiece& p) {
    const float2 a = unpack_f2(p.lo), b = unpack_f2(p.hi);
    return make_float4(a.x, a.y, b.x, b.y);
}
// S <- exp(dt A) S + dx B for four elements; y gains their S C, pair by pair.
__device__ __forceinline__ void mamba_update(ScanPiece& S, const ScanPiece& A, const ScanPiece& B, const ScanPiece& C, f32x2 dt, f32x2 dx, f32x2& y) {
    S.lo = fma2(decay_m1(mul2(dt, A.lo)), S.lo, fma2(dx, B.lo, S.lo));
    S.hi = fma2(decay_m1(mul2(dt, A.hi)), S.hi, fma2(dx, B.hi, S.hi));
    y = fma2(S.lo, C.lo, y);
    y = fma2(S.hi, C.hi, y);
}
__device__ __forceinline__ float pair_sum(f32x2 v) {
    const float2 f = unpack_f2(v);
    return f.x + f.y;
}
template <int L>
__device__ __forceinline__ float lane_group_sum(float v) {
#pragma unroll
    for (int o = L / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
// Where element i of a token's padded dt | B | C row (dt to dt_pitch, B and C to state_pitch) lies in the unpadded one; -1 =
// padding.
__device__ __forceinline__ int mamba_low_source(const MambaScanArgs& a, int i) {
    if (i < a.dt_pitch) return i < a.dt_rank ? i : -1;
    i -= a.dt_pitch;
    const int from = i < a.state_pitch ? a.dt_rank : a.dt_rank + a.state;
    if (i >= a.state_pitch) i -= a.state_pitch;
    return i < a.state ? from + i : -1;
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
    constexpr int pieces = L * NS;
    const int vecs = a.dt_pitch / kVec;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    const float4* A4 = reinterpret_cast<const float4*>(a.A) + (size_t)(in ? c : 0) * pieces + ln;
    float4* S4 = reinterpret_cast<float4*>(a.S) + (size_t)(in ? c : 0) * pieces + ln;
    ScanPiece A[NS], S[NS];
#pragma unroll
    for (int i = 0; i < NS; ++i) {
        A[i] = scan_piece(__ldg(A4 + i * L));
        S[i] = scan_piece(pos > 0 ? __ldcg(S4 + i * L) : zero);
    }
    const uint4* w = reinterpret_cast<const uint4*>(reinterpret_cast<const WT*>(a.w_dt) + (size_t)(in ? c : 0) * a.dt_pitch);
    uint4 wv[kAhead];
#pragma unroll
    for (int i = 0; i < kAhead; ++i)
        if (ln + i * L < vecs) wv[i] = ldg_stream_u4(w + ln + i * L);
    const float bias = in ? __ldg(a.dt_b + c) : 0.f, D = in ? __ldg(a.D + c) : 0.f;
    pdl_wait();
    const float x = in ? __ldcg(a.x + c) : 0.f, z = in ? __ldcg(a.z + c) : 0.f;
    for (int i = tid; i < a.dt_pitch + 2 * a.state_pitch; i += kScanStepThreads) {
        const int src = mamba_low_source(a, i);
        const float v = __ldcg(a.low + max(src, 0));
        sc_low[i] = src >= 0 ? v : 0.f;
    }
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
    f32x2 y2 = both(0.f);
#pragma unroll
    for (int i = 0; i < NS; ++i) mamba_update(S[i], A[i], scan_piece(B[ln + i * L]), scan_piece(C[ln + i * L]), both(dt), both(dt * x), y2);
    const float y = lane_group_sum<L>(pair_sum(y2));
    if (!in || !ok) return;
#pragma unroll
    for (int i = 0; i < NS; ++i) S4[i * L] = scan_float4(S[i]);
    if (ln == 0) a.out[c] = fmaf(D, x, y) * z;
}

}  // namespace lpp
