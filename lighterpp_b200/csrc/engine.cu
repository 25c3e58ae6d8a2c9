// Host side of the B200 decode engine: device memory layout, weight repacking, the per-token
// CUDA graph and the C ABI declared in include/lpp_b200.h.
//
// Stands in for the device halves of malloc_run_state / free_run_state (src/model.cpp:18-118),
// attention / transformer_block / forward (src/model.cpp:121-384, USE_CUDA branches) and the upload
// code of the loaders (src/loader.cpp:73-131, 543-637) of the reference tree.
//
// Device layout (per tensor-parallel rank; Dq = local query rows, KVd = local kv rows, Fl = local
// FFN columns):
//   wqkv [L][Dq + 2*KVd][D]   rows q | k | v of one layer back to back  -> one fused GEMV
//   wo   [L][D][Dq]           column slice of the reference wo, repacked contiguous
//   w13  [L][2*Fl][D]         gate row i and up row i interleaved         -> SwiGLU in the epilogue
//   w2   [L][D][Fl]           column slice of the reference w2
//   emb / wcls [V][D]         weight dtype; wcls aliases emb when the classifier is tied
//   K, V cache [L][KVHl][S][hs]   FP16 (or FP32), the reference's index order
//   rope [S][hs/2] (cos, sin)     built on the host with libm so rotations match the CPU path bit
//                                 for bit
// Engines made by lpp_engine_create_layers keep one allocation per matrix and layer (ModelLayer below): layers may
// differ in mixer and in every size, rows are padded with zeros to a multiple of 64 inputs.  What a sequence leaves behind
// (cache rows, recurrent state) belongs to a run of a layer (LayerRun): a layer inside the loop has one per pass.
#include <cuda_runtime.h>
#include <cuda_fp16.h>
#include <dlfcn.h>
#include <math.h>
#include <stdarg.h>
#include <stdio.h>
#include <stdlib.h>
#include <string.h>

#include <algorithm>
#include <string>
#include <vector>

#include "../../include/lpp_b200.h"
#include "attention.cuh"
#include "common.cuh"
#include "gemv.cuh"
#include "latent_attention.cuh"
#include "mamba.cuh"
#include "ops.cuh"
#include "prefill.cuh"
#include "prefill_mixers.cuh"
#include "sampler.cuh"
#include "sampler_exact.cuh"
#include "shared_kv.cuh"

using namespace lpp;

// ------------------------------------------------------------------ error plumbing

static thread_local std::string g_err;
static lpp_status fail(lpp_status s, const char* fmt, ...) {
    char buf[512];
    va_list ap;
    va_start(ap, fmt);
    vsnprintf(buf, sizeof buf, fmt, ap);
    va_end(ap);
    g_err = buf;
    return s;
}
void lpp_internal_set_error(const char* msg) { g_err = msg ? msg : ""; }
#define CU(call)                                                                                   \
    do {                                                                                           \
        cudaError_t e_ = (call);                                                                   \
        if (e_ != cudaSuccess)                                                                     \
            return fail(LPP_ERR_CUDA, "%s failed: %s (%s:%d)", #call, cudaGetErrorString(e_), __FILE__, __LINE__); \
    } while (0)
#define TRY(call)                      \
    do {                               \
        lpp_status s_ = (call);        \
        if (s_ != LPP_OK) return s_;   \
    } while (0)

// Timing aids: environment switches that change what a step launches (kernel kinds left out, arithmetic
// skipped, stage sizes, prefetch depth ...).  Some make the results meaningless, so they exist only in
// builds made with -DLPP_TIMING_AIDS; the product build never looks at them.
#ifdef LPP_TIMING_AIDS
static const char* aid_env(const char* name) { return getenv(name); }
#else
static const char* aid_env(const char*) { return nullptr; }
#endif

// LPP_TRACE=1 in the environment prints one line per host-side phase and synchronises after every
// launch of an un-graphed step, to localise a failing kernel.
static bool tracing() {
    static int t = -1;
    if (t < 0) t = getenv("LPP_TRACE") ? 1 : 0;
    return t == 1;
}
#define TRACE(...)                        \
    do {                                  \
        if (tracing()) {                  \
            fprintf(stderr, "[lpp] " __VA_ARGS__); \
            fprintf(stderr, "\n");        \
            fflush(stderr);               \
        }                                 \
    } while (0)

// ------------------------------------------------------------------ NCCL through dlopen
// Only tensor-parallel engines need NCCL, so it is bound at run time; a single-GPU process never
// loads it.  The handful of prototypes below follow nccl.h.

namespace nccl {
typedef struct ncclComm* comm_t;
typedef struct { char internal[128]; } unique_id;
typedef int result_t;
static void* lib = nullptr;
static result_t (*GetUniqueId)(unique_id*);
static result_t (*CommInitRank)(comm_t*, int, unique_id, int);
static result_t (*CommDestroy)(comm_t);
static result_t (*AllReduce)(const void*, void*, size_t, int /*dtype*/, int /*op*/, comm_t, cudaStream_t);
static const char* (*GetErrorString)(result_t);
constexpr int kFloat32 = 7, kSum = 0;
static bool load() {
    if (lib) return true;
    const char* names[] = {"libnccl.so.2", "libnccl.so"};
    for (const char* n : names) {
        lib = dlopen(n, RTLD_NOW | RTLD_GLOBAL);
        if (lib) break;
    }
    if (!lib) return false;
    GetUniqueId = (decltype(GetUniqueId))dlsym(lib, "ncclGetUniqueId");
    CommInitRank = (decltype(CommInitRank))dlsym(lib, "ncclCommInitRank");
    CommDestroy = (decltype(CommDestroy))dlsym(lib, "ncclCommDestroy");
    AllReduce = (decltype(AllReduce))dlsym(lib, "ncclAllReduce");
    GetErrorString = (decltype(GetErrorString))dlsym(lib, "ncclGetErrorString");
    return GetUniqueId && CommInitRank && CommDestroy && AllReduce && GetErrorString;
}
}  // namespace nccl

// ------------------------------------------------------------------ engine

enum Kind { kQkv = 0, kAttn = 1, kOproj = 2, kGateUp = 3, kDown = 4, kLmHead = 5, kSampler = 6, kAllReduce = 7, kLatQuery = 8, kLatValue = 9, kScanIn = 10, kScan = 11, kKinds = 12 };

// One layer of an engine described layer by layer.  Weight matrices: rows x pitch, pitch = inputs rounded up to 64, zero
// padded; element type = weight_dtype.
struct ModelLayer {
    lpp_layer_desc d;
    int in_rows;                // rows of the input matrix: everything the mixer projects its input with
    int o_in, o_pitch, ff_pitch;  // inputs of the output projection, and of it and the down projection with padding
    void *w_in = nullptr, *wo = nullptr, *w13 = nullptr, *w2 = nullptr;
    float *n1w = nullptr, *n1b = nullptr, *n2w = nullptr, *n2b = nullptr, *o_b = nullptr;
    CUtensorMap m_in, m_wo, m_w13, m_w2, x_att, x_hb;   // weights, activation blocks with this layer's widths (batched path)
    // attention over shared rows (latent_attention.cuh): heads of a group, groups, value part and whole of a row
    int group_heads = 0, groups = 0, rank_pitch = 0, row_width = 0;
    const float2* rope = nullptr;
    // latent attention (latent.cuh)
    int dim_pitch, val_pitch;   // inputs per head of the query and of the value matrix
    int vdim_rows;              // rows per head of the value matrix
    int q_plain_rows, q_rot_rows, latent_rows;
    void *w_uk = nullptr, *w_uv = nullptr;
    float* lat_w = nullptr;
    CUtensorMap m_uk, m_uv, x_qn, x_olat;
    // attention whose values are its keys (shared_kv.cuh)
    int head_rows, q_rows, k_rows;
    float* qk_b = nullptr;
    // selective scan (mamba.cuh)
    int inner_rows, inner_pitch, low_rows, dt_pitch, state_pitch;
    void *w_low = nullptr, *w_dt = nullptr;
    float *conv_w = nullptr, *conv_b = nullptr, *dt_b = nullptr, *A = nullptr, *skip = nullptr;
    CUtensorMap m_low, x_low;
};
// A layer in its place in the order of execution, with what it keeps of the sequence.
struct LayerRun {
    int layer;
    int step_row = -1;          // row of the loop's vectors that is added before this run, -1 = none
    void* cache = nullptr;      // [groups][seq_len][row_width]
    float* ring = nullptr;      // convolution inputs [taps - 1][inner_rows]
    float* S = nullptr;         // recurrent state [inner][state_pitch]
    // vectors added with the output and with the down projection: the output's bias, and the loop's vector that comes before
    // the next run (with the last of the two products); nullptr = none
    const float *o_add = nullptr, *down_add = nullptr;
    float* sum_add = nullptr;   // storage of their sum where there are both
};

struct lpp_engine {
    lpp_config c;
    int hs, Hl, KVHl, Dq, KVd, Fl, gqa;
    int esz, kvesz;
    int num_sms;
    int attn_splits, attn_gb, attn_z;
    int attn_splits_long;  // splits of the tensor-core kernel: one CTA per SM, one wave
    int sample_blocks;
    size_t smem_optin;
    cudaStream_t stream = nullptr;
    // weights
    void *wqkv = nullptr, *wo = nullptr, *w13 = nullptr, *w2 = nullptr, *emb = nullptr, *wcls = nullptr;
    float *rms_att = nullptr, *rms_ffn = nullptr, *rms_final = nullptr, *final_b = nullptr;
    // norms: RMS with the reference's epsilon unless the model says otherwise; Dp = width of a row in memory
    int Dp = 0, Vp = 0;  // row pitch of width-sized vectors, classifier rows
    bool layer_norm = false;
    float norm_eps = 1e-5f;  // src/ops.cpp:20-32
    // layers of lpp_engine_create_layers (empty for the reference's own architecture), buffers their steps share
    std::vector<ModelLayer> layers;
    std::vector<LayerRun> runs;
    float emb_scale = 1.f, logit_scale = 1.f;  // the latter is part of the final norm's weight and bias on the device
    float* loop_vec = nullptr;                 // [loop_rows][Dp]
    int loop_rows = 0;
    // Tokens of the sequence that the recurrent state has seen (a cache can be rewritten from any position, a state goes on
    // from where it stands or starts anew), -1 = unknown.  Stays 0 without recurrent layers.
    bool recurrent = false;
    int state_len = 0;
    float *scan_x = nullptr, *scan_z = nullptr, *scan_low = nullptr;
    unsigned int* row_counters = nullptr;
    std::vector<std::pair<lpp_layer_desc, float2*>> rope_tables;
    float *lat_qplain = nullptr, *lat_raw = nullptr, *lat_gate = nullptr, *lat_part = nullptr;
    void* lat_query = nullptr;
    bool wcls_owned = false;
    bool wcls_shard_only = false;  // an untied classifier of a tensor-parallel rank holds this rank's vocabulary rows only
    std::vector<unsigned char> got;  // upload bookkeeping: [tensor][layer]
    // state
    void *kcache = nullptr, *vcache = nullptr;
    float *xa = nullptr, *xb = nullptr, *q = nullptr, *att_out = nullptr, *hb = nullptr, *logits = nullptr;
    float *attn_part = nullptr, *samp_max = nullptr, *samp_sum = nullptr, *r_values = nullptr;
    int *samp_idx = nullptr, *out_tokens = nullptr;
    unsigned int *attn_counters = nullptr, *samp_counter = nullptr;
    // exact-order sampler scratch
    bool exact_sampler = false;
    unsigned int* ex_sync = nullptr;
    double* ex_block_sum = nullptr;
    int* ex_entry_count = nullptr;
    ExactEntry* ex_entries = nullptr;
    float* ex_scalars = nullptr;
    float2* rope = nullptr;
    StepState* st = nullptr;
    int run_cap = 0;  // capacity of r_values / out_tokens
    // host staging (pinned)
    StepState* h_st = nullptr;
    int* h_out = nullptr;  // out_token, status
    // upload staging
    void* stage = nullptr;
    size_t stage_bytes = 0;
    // tensor-parallel exchange over peer memory: per exchange (2 per layer) a receive area [tp][dim] floats
    // and two counters; peer_base[p] = rank p's buffer as mapped into this process (own buffer for p == rank)
    unsigned char* tp_buf = nullptr;
    size_t tp_buf_bytes = 0;
    unsigned char* peer_base[kMaxTp] = {};
    bool peer_ready = false;
    unsigned char* absent_peer = nullptr;  // test aid: where stores to ranks that do not exist go (lpp_debug_tp_absent_peers)
    unsigned long long* gtrace = nullptr;  // LPP_GEMV_TRACE: per-launch per-CTA time stamps of the ring GEMV
    // graphs
    // graph variants by context length; only [0] is used at present
    cudaGraphExec_t g_full[2] = {nullptr, nullptr}, g_logits[2] = {nullptr, nullptr};

    // batched prompt path (allocated by the first lpp_prefill)
    float *pf_x = nullptr, *pf_q = nullptr, *pf_part = nullptr;
    void *pf_xn = nullptr, *pf_att = nullptr, *pf_hb = nullptr;
    int *pf_tokens = nullptr, *pf_rows = nullptr;
    float* pf_logits = nullptr;
    CUtensorMap pf_map_cls;
    void *pf_qn = nullptr, *pf_olat = nullptr;      // latent attention: plain queries, attended latents (hi + lo operands)
    __half* pf_lq = nullptr;                        // query rows
    float *pf_lpart = nullptr, *pf_gate = nullptr;  // attention partials, gates
    float *pf_sx = nullptr, *pf_sz = nullptr, *pf_tail = nullptr;  // selective scan: convolved x, z, last convolution inputs
    float* pf_low = nullptr;                                       // dt | B | C rows
    void* pf_sxp = nullptr;                                        // x as hi + lo operands
    CUtensorMap pf_map_wqkv, pf_map_wo, pf_map_w13, pf_map_w2, pf_map_xn, pf_map_att, pf_map_hb;
    bool pf_ready = false;

    bool finalized = false;
    int kernels_full = 0;
    cudaEvent_t ev0 = nullptr, ev1 = nullptr;
    // NCCL
    nccl::comm_t comm = nullptr;
    // profiling hooks
    bool profiling = false;
    bool profiling_capture = false;
    int only_kind = -1;  // lpp_profile_kind: the one kind recorded
    std::vector<cudaEvent_t> prof_events;
    std::vector<int> prof_kinds;
};

static size_t align_up(size_t v, size_t a) { return (v + a - 1) / a * a; }

template <typename... KArgs, typename... Args>
static cudaError_t launch_clusters(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t s,
                                   bool pdl, int cluster_x, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = s;
    cudaLaunchAttribute attr[2];
    cfg.attrs = attr;
    cfg.numAttrs = 0;
    if (pdl) {
        attr[cfg.numAttrs].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[cfg.numAttrs++].val.programmaticStreamSerializationAllowed = 1;
    }
    if (cluster_x > 0) {  // CTAs of a cluster, along x
        attr[cfg.numAttrs].id = cudaLaunchAttributeClusterDimension;
        attr[cfg.numAttrs].val.clusterDim.x = (unsigned)cluster_x;
        attr[cfg.numAttrs].val.clusterDim.y = 1;
        attr[cfg.numAttrs++].val.clusterDim.z = 1;
    }
    return cudaLaunchKernelEx(&cfg, kernel, args...);
}
template <typename... KArgs, typename... Args>
static cudaError_t launch_kernel(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t s,
                                 bool pdl, Args... args) {
    return launch_clusters(kernel, grid, block, smem, s, pdl, 0, args...);
}

// ---- GEMV dispatch

struct GemvPlan {
    dim3 grid;
    int threads;
    size_t smem;
};

constexpr int kStageTarget = 8192;  // bytes per bulk copy / ring slot (see gemv.cuh)

// A stage is one bulk copy of about stage_target bytes: whole row pairs when they fit, else one
// K-chunk of one row.
static void gemv_geometry(GemvArgs& a, int esz, int stage_target) {
    const int pair_bytes = kRowsPerGroup * a.K * esz;
    if (pair_bytes <= stage_target) {
        a.pairs_per_stage = stage_target / pair_bytes;
        a.kc = a.K;
        a.stage_bytes = a.pairs_per_stage * pair_bytes;
    } else {
        a.pairs_per_stage = 0;
        a.kc = std::max(8, std::min(a.K, stage_target / esz) / 8 * 8);
        a.stage_bytes = a.kc * esz;
    }
}

template <typename WT, int EPI, bool LN = false>
static cudaError_t launch_gemv_t(lpp_engine* e, GemvArgsOf<EPI>& a, bool pdl, cudaStream_t s) {
    const int esz = sizeof(WT);
    const int groups = a.n_rows / kRowsPerGroup;
    // Grouped rows: a CTA stages the inputs of every group its contiguous row pairs touch, plus the split weights.
    auto staged_bytes = [&](int grid) -> size_t {
        if (a.group_pairs <= 0) return align_up((size_t)a.K * 4, 128);
        const int pairs = (groups + grid - 1) / grid;  // grid: CTAs with rows
        const size_t n = (size_t)(pairs + a.group_pairs - 2) / a.group_pairs + 1;
        return align_up(n * ((size_t)a.K + kLatentMaxSplits) * 4, 128);
    };
    if (e->c.flags & LPP_FLAG_GEMV_LDG) {
        const size_t smem = 128 + staged_bytes(std::max(1, std::min(groups, e->num_sms * 4)));
        static bool attr_done[64] = {};
        if (!attr_done[e->c.device & 63]) {
            cudaError_t r = cudaFuncSetAttribute(gemv_ldg_kernel<WT, EPI, LN>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                 (int)e->smem_optin);
            if (r != cudaSuccess) return r;
            attr_done[e->c.device & 63] = true;
        }
        const int grid = std::max(1, std::min(groups, e->num_sms * 4)) + (EPI == kEpiLatentQuery ? 1 : 0);
        return launch_kernel(gemv_ldg_kernel<WT, EPI, LN>, dim3(grid), dim3(kGemvLdgThreads), smem, s, pdl, a);
    }
    // LPP_STAGE_KB (timing experiments) overrides the 8 KiB stage size.
    int stage_target = kStageTarget;
    if (const char* sk = aid_env("LPP_STAGE_KB")) stage_target = std::max(1, atoi(sk)) * 1024;
    gemv_geometry(a, esz, stage_target);
    // the query GEMV of latent attention: one CTA without rows (row_ctas in gemv.cuh)
    const int extra = EPI == kEpiLatentQuery ? 1 : 0;
    const int grid = std::max(1, std::min(groups, e->num_sms - extra));
    const size_t xbytes = staged_bytes(grid);
    a.xs_bytes = (int)xbytes;
    const size_t fixed = kGemvBarrierBytes + 128 + xbytes;
    if (fixed >= e->smem_optin) return cudaErrorInvalidValue;
    size_t ring = (size_t)(e->c.ring_kb > 0 ? e->c.ring_kb : 128) * 1024;
    if (fixed + ring > e->smem_optin) ring = e->smem_optin - fixed;
    int ns = (int)(ring / ((size_t)kGemvConsumerWarps * a.stage_bytes));  // slots per consumer warp
    ns = std::max(2, std::min(ns, kGemvMaxStages));
    a.n_stages = ns;
    const size_t smem = fixed + (size_t)kGemvConsumerWarps * ns * a.stage_bytes;
    if (smem > e->smem_optin) return cudaErrorInvalidValue;
    static bool attr_done[64] = {};
    if (!attr_done[e->c.device & 63]) {
        cudaError_t r = cudaFuncSetAttribute(gemv_ring_kernel<WT, EPI, LN>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                             (int)e->smem_optin);
        if (r != cudaSuccess) return r;
        attr_done[e->c.device & 63] = true;
    }
    return launch_kernel(gemv_ring_kernel<WT, EPI, LN>, dim3(grid + extra), dim3(kGemvRingThreads), smem, s, pdl, a);
}

static cudaError_t launch_gemv(lpp_engine* e, int epi, int w_dtype, GemvArgs& a, bool pdl, cudaStream_t s) {
#define LPP_GEMV_CASE(E)                                                                                                \
    case E:                                                                                                             \
        if (w_dtype == LPP_BF16) return launch_gemv_t<__nv_bfloat16, E>(e, a, pdl, s);                                  \
        return w_dtype == LPP_F16 ? launch_gemv_t<__half, E>(e, a, pdl, s) : launch_gemv_t<float, E>(e, a, pdl, s);
#define LPP_GEMV_LN_CASE(E)                                                                                             \
    case E:                                                                                                             \
        return w_dtype == LPP_BF16 ? launch_gemv_t<__nv_bfloat16, E, true>(e, a, pdl, s) : launch_gemv_t<float, E, true>(e, a, pdl, s);
    if (a.norm_b) {
        switch (epi) {
            LPP_GEMV_LN_CASE(kEpiStore)
            LPP_GEMV_LN_CASE(kEpiSwiglu)
        }
        return cudaErrorInvalidValue;
    }
    switch (epi) {
        LPP_GEMV_CASE(kEpiStore)
        LPP_GEMV_CASE(kEpiResid)
        LPP_GEMV_CASE(kEpiSwiglu)
        case kEpiResidBias:
            return w_dtype == LPP_BF16 ? launch_gemv_t<__nv_bfloat16, kEpiResidBias>(e, a, pdl, s) : launch_gemv_t<float, kEpiResidBias>(e, a, pdl, s);
        case kEpiQkv:
            return w_dtype == LPP_F16 ? launch_gemv_t<__half, kEpiQkv>(e, a, pdl, s) : launch_gemv_t<float, kEpiQkv>(e, a, pdl, s);
    }
#undef LPP_GEMV_CASE
#undef LPP_GEMV_LN_CASE
    return cudaErrorInvalidValue;
}
template <int EPI, bool LN>
static cudaError_t launch_latent_gemv(lpp_engine* e, int w_dtype, GemvLatentArgs& a, bool pdl, cudaStream_t s) {
    return w_dtype == LPP_BF16 ? launch_gemv_t<__nv_bfloat16, EPI, LN>(e, a, pdl, s) : launch_gemv_t<float, EPI, LN>(e, a, pdl, s);
}
static cudaError_t launch_gemv(lpp_engine* e, int epi, int w_dtype, GemvLatentArgs& a, bool pdl, cudaStream_t s) {
    switch (epi) {
        case kEpiLatentIn:
            return a.norm_b ? launch_latent_gemv<kEpiLatentIn, true>(e, w_dtype, a, pdl, s) : launch_latent_gemv<kEpiLatentIn, false>(e, w_dtype, a, pdl, s);
        case kEpiLatentQuery: return launch_latent_gemv<kEpiLatentQuery, false>(e, w_dtype, a, pdl, s);
        case kEpiLatentValue: return launch_latent_gemv<kEpiLatentValue, false>(e, w_dtype, a, pdl, s);
    }
    return cudaErrorInvalidValue;
}
// Input projections with a row epilogue.
template <int EPI>
static cudaError_t launch_row_gemv(lpp_engine* e, int w_dtype, GemvArgsOf<EPI>& a, bool pdl, cudaStream_t s) {
    if (w_dtype == LPP_BF16)
        return a.norm_b ? launch_gemv_t<__nv_bfloat16, EPI, true>(e, a, pdl, s) : launch_gemv_t<__nv_bfloat16, EPI, false>(e, a, pdl, s);
    return a.norm_b ? launch_gemv_t<float, EPI, true>(e, a, pdl, s) : launch_gemv_t<float, EPI, false>(e, a, pdl, s);
}
static cudaError_t launch_gemv(lpp_engine* e, int, int w_dtype, GemvSharedKvArgs& a, bool pdl, cudaStream_t s) {
    return launch_row_gemv<kEpiSharedKvIn>(e, w_dtype, a, pdl, s);
}
static cudaError_t launch_gemv(lpp_engine* e, int, int w_dtype, GemvMambaArgs& a, bool pdl, cudaStream_t s) {
    return launch_row_gemv<kEpiMambaIn>(e, w_dtype, a, pdl, s);
}

// ---- attention dispatch

template <typename KT, int DPL>
static cudaError_t launch_attn_d(lpp_engine* e, const AttnArgs& a, dim3 grid, bool pdl, cudaStream_t s) {
    switch (e->attn_gb) {
        case 4:
            return launch_kernel(attn_decode_kernel<KT, DPL, 4>, grid, dim3(kAttnKernelThreads), 0, s, pdl, a);
        case 2:
            return launch_kernel(attn_decode_kernel<KT, DPL, 2>, grid, dim3(kAttnKernelThreads), 0, s, pdl, a);
        default:
            return launch_kernel(attn_decode_kernel<KT, DPL, 1>, grid, dim3(kAttnKernelThreads), 0, s, pdl, a);
    }
}
template <typename KT>
static cudaError_t launch_attn_t(lpp_engine* e, const AttnArgs& a, dim3 grid, bool pdl, cudaStream_t s) {
    switch (e->hs / 8) {
        case 2: return launch_attn_d<KT, 2>(e, a, grid, pdl, s);
        case 4: return launch_attn_d<KT, 4>(e, a, grid, pdl, s);
        case 6: return launch_attn_d<KT, 6>(e, a, grid, pdl, s);
        case 8: return launch_attn_d<KT, 8>(e, a, grid, pdl, s);
        case 12: return launch_attn_d<KT, 12>(e, a, grid, pdl, s);
        case 16: return launch_attn_d<KT, 16>(e, a, grid, pdl, s);
    }
    return cudaErrorInvalidValue;
}

// Attention with the scores and P.V on the tensor cores (FP16 cache, head size 64 or 128, 1/2/4/8 query heads
// per KV head); other shapes keep the CUDA-core kernel.
static cudaError_t launch_attn_mma(lpp_engine* e, const AttnArgs& a, bool pdl, cudaStream_t s) {
    if (e->c.kv_dtype != LPP_F16) return cudaErrorNotSupported;
    const dim3 grid(a.n_splits, e->KVHl, 1), block(kAttnKernelThreads);
#define LPP_MMA_CASE(HS_, G_) \
    if (e->hs == HS_ && e->gqa == G_) return launch_kernel(attn_mma_kernel<HS_, G_>, grid, block, 0, s, pdl, a);
    LPP_MMA_CASE(64, 1) LPP_MMA_CASE(64, 2) LPP_MMA_CASE(64, 4) LPP_MMA_CASE(64, 8)
    LPP_MMA_CASE(128, 1) LPP_MMA_CASE(128, 2) LPP_MMA_CASE(128, 4) LPP_MMA_CASE(128, 8)
#undef LPP_MMA_CASE
    return cudaErrorNotSupported;
}
static bool attn_mma_supported(const lpp_engine* e) {
    return e->c.kv_dtype == LPP_F16 && (e->hs == 64 || e->hs == 128) && (e->gqa == 1 || e->gqa == 2 || e->gqa == 4 || e->gqa == 8);
}

// ---- latent attention: the tensor-core kernel where query and key tiles fit shared memory, else the CUDA-core kernel

constexpr int kLatStepWarps = 8, kLatBlockWarps = 16;  // warps of an attention CTA: one token, prompt block
constexpr int kLatMinChunk = 64;       // fewest keys worth a split of their own when splits are left apart
constexpr int kLatClusterChunk = 32;   // ... when they meet in a cluster (prompt blocks)
constexpr int kLatClusterKeys = 8192;  // spans beyond this take more splits than a cluster holds

static bool latent_mma_supported(const lpp_engine* e, const ModelLayer& y) {
    return e->c.kv_dtype == LPP_F16 && y.rank_pitch <= 512 && (size_t)latent_mma_smem<1, kLatBlockWarps>(y.row_width) <= e->smem_optin &&
           !(e->c.flags & LPP_FLAG_LATENT_CUDA_CORES);
}
// How an attention launch of n_tokens is laid out: rows per tile, splits of the keys, whether the splits are a cluster.
struct LatentPlan {
    bool mma;
    int tile_rows, splits, min_chunk;
    bool cluster;
};
static LatentPlan latent_plan(const lpp_engine* e, const ModelLayer& y, int n_tokens) {
    LatentPlan p = {};
    const int heads = y.group_heads, rows = n_tokens * heads;  // of a group
    p.mma = latent_mma_supported(e, y);
    // one token: tiles of 16 heads, so that as many CTAs as possible share the keys; a prompt block: 32 rows
    p.tile_rows = !p.mma ? 1 : (n_tokens == 1 || rows <= 16 || (size_t)latent_mma_smem<2, kLatBlockWarps>(y.row_width) > e->smem_optin) ? 16 : 32;
    const int tiles = (rows + p.tile_rows - 1) / p.tile_rows * y.groups;
    const int tile_tokens = n_tokens == 1 ? 1 : std::min(n_tokens, (p.tile_rows - 1) / heads + 2);
    const int keys = std::min(e->c.seq_len, y.d.window > 0 ? y.d.window + tile_tokens - 1 : e->c.seq_len);
    p.cluster = p.mma && n_tokens > 1 && keys <= kLatClusterKeys;
    p.min_chunk = p.cluster ? kLatClusterChunk : kLatMinChunk;
    const int fill = n_tokens > 1 ? std::max(1, e->num_sms / tiles) : y.groups == 1 ? kLatentMaxSplits : std::max(1, 2 * e->num_sms / tiles);
    p.splits = std::max(1, std::min({kLatentMaxSplits, (keys + p.min_chunk - 1) / p.min_chunk, fill}));
    if (p.cluster) p.splits = p.splits >= kLatentMaxCluster ? kLatentMaxCluster : p.splits >= 4 ? 4 : p.splits >= 2 ? 2 : 1;
    return p;
}

template <int MT, int NT, int NW, bool SKV>
static cudaError_t launch_latent_mma_t(lpp_engine* e, const LatentAttnArgs& a, int splits, bool pdl, cudaStream_t s) {
    static bool attr_done[64] = {};
    if (!attr_done[e->c.device & 63]) {
        const cudaError_t r = cudaFuncSetAttribute(latent_attn_mma_kernel<MT, NT, NW, SKV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)e->smem_optin);
        if (r != cudaSuccess) return r;
        attr_done[e->c.device & 63] = true;
    }
    const dim3 grid(splits, (a.n_tokens * a.heads + 16 * MT - 1) / (16 * MT), a.all_heads / a.heads);
    return launch_clusters(latent_attn_mma_kernel<MT, NT, NW, SKV>, grid, dim3(32 * NW), (size_t)latent_mma_smem<MT, NW>(a.row_width), s, pdl,
                           a.cluster ? splits : 0, a);
}
template <int MT, int NT, int NW>
static cudaError_t launch_latent_mma(lpp_engine* e, const LatentAttnArgs& a, int splits, bool skv, bool pdl, cudaStream_t s) {
    return skv ? launch_latent_mma_t<MT, NT, NW, true>(e, a, splits, pdl, s) : launch_latent_mma_t<MT, NT, NW, false>(e, a, splits, pdl, s);
}
static cudaError_t launch_latent_attn(lpp_engine* e, const LatentPlan& p, const LatentAttnArgs& a, bool skv, bool pdl, cudaStream_t s) {
    const int rp = a.rank_pitch;
    if (p.mma) {
        constexpr int S = kLatStepWarps, B = kLatBlockWarps;
        if (a.n_tokens == 1)
            return rp <= 128   ? launch_latent_mma<1, 2, S>(e, a, p.splits, skv, pdl, s)
                   : rp <= 256 ? launch_latent_mma<1, 4, S>(e, a, p.splits, skv, pdl, s)
                               : launch_latent_mma<1, 8, S>(e, a, p.splits, skv, pdl, s);
        if (p.tile_rows == 16)
            return rp <= 256 ? launch_latent_mma<1, 2, B>(e, a, p.splits, skv, pdl, s) : launch_latent_mma<1, 4, B>(e, a, p.splits, skv, pdl, s);
        return rp <= 256 ? launch_latent_mma<2, 2, B>(e, a, p.splits, skv, pdl, s) : launch_latent_mma<2, 4, B>(e, a, p.splits, skv, pdl, s);
    }
    const dim3 grid(p.splits, a.all_heads, a.n_tokens);
    // query row and scores of a tile, or what one row's combination needs
    const size_t smem = (size_t)std::max(a.row_width + kLatentTile, kLatentMaxSplits + 4 * kLatentThreads) * 4;
    if (e->c.kv_dtype == LPP_F32) return launch_kernel(latent_attn_kernel<float>, grid, dim3(kLatentThreads), smem, s, pdl, a);
    return launch_kernel(latent_attn_kernel<__half>, grid, dim3(kLatentThreads), smem, s, pdl, a);
}
static LatentArgs latent_args(const lpp_engine* e, const ModelLayer& y, const LayerRun& r) {
    LatentArgs L = {};
    L.heads = y.d.heads;
    L.dim = y.d.dim;
    L.rot = y.d.rot_dim;
    L.vdim = y.d.vdim;
    L.rank = y.d.kv_rank;
    L.dim_pitch = y.dim_pitch;
    L.rank_pitch = y.rank_pitch;
    L.row_width = y.row_width;
    L.vdim_rows = y.vdim_rows;
    L.q_plain_rows = y.q_plain_rows;
    L.q_rot_rows = y.q_rot_rows;
    L.latent_rows = y.latent_rows;
    L.cache_f32 = e->c.kv_dtype == LPP_F32;
    L.rope = y.rope;
    L.q_plain = e->lat_qplain;
    L.latent = e->lat_raw;
    L.gate = e->lat_gate;
    L.query = e->lat_query;
    L.cache = r.cache;
    L.norm_w = y.lat_w;
    L.norm_eps = e->norm_eps;
    L.part = e->lat_part;
    const LatentPlan p = latent_plan(e, y, 1);
    L.window = y.d.window;
    L.max_splits = p.splits;
    L.min_chunk = p.min_chunk;
    return L;
}
// For one token; a prompt block overrides what differs.
static LatentAttnArgs latent_attn_args(const lpp_engine* e, const ModelLayer& y, const LayerRun& r, const LatentPlan& p) {
    LatentAttnArgs a = {};
    a.cluster = p.cluster;
    a.q = e->lat_query;
    a.cache = r.cache;
    a.part = e->lat_part;
    a.st = e->st;
    a.start_pos = -1;
    a.n_tokens = 1;
    a.heads = y.group_heads;
    a.all_heads = y.group_heads * y.groups;
    a.rank_pitch = y.rank_pitch;
    a.row_width = y.row_width;
    if (y.d.mixer == LPP_MIXER_LATENT) {
        a.plane_pitch = y.val_pitch;
        a.plane_cols = y.rank_pitch;
        a.plane_row = y.d.heads * y.val_pitch;
    } else {  // finished rows are the output projection's input
        a.plane_pitch = a.plane_cols = a.out_cols = y.d.dim;
        a.plane_row = y.o_pitch;
        a.score_skip = y.d.rot_dims / 16;
        a.softcap = y.d.softcap;
        a.cap_rate = y.d.softcap > 0.f ? 2.f / y.d.softcap : 0.f;
        a.out = e->att_out;
        a.gate = y.d.gate ? e->lat_gate : nullptr;
        a.counters = e->row_counters;
    }
    a.window = y.d.window;
    a.max_splits = p.splits;
    a.min_chunk = p.min_chunk;
    a.seq_len = e->c.seq_len;
    a.scale = y.d.scale;
    return a;
}

// ---- attention whose values are its keys, selective scan

// Constants and state may be read ahead of a step kernel's dependency wait when steps are separate graph launches: what
// earlier steps wrote is then complete.
static int step_early(const lpp_engine* e) { return (e->c.flags & LPP_FLAG_NO_GRAPH) ? 0 : 1; }

static SharedKvArgs shared_kv_args(const lpp_engine* e, const ModelLayer& y, const LayerRun& r) {
    SharedKvArgs s = {};
    s.heads = y.d.heads;
    s.kv_heads = y.d.kv_heads;
    s.dim = y.d.dim;
    s.rot = y.d.rot_dims;
    s.head_rows = y.head_rows;
    s.q_rows = y.q_rows;
    s.k_rows = y.k_rows;
    s.rank_pitch = y.rank_pitch;
    s.row_width = y.row_width;
    s.cache_f32 = e->c.kv_dtype == LPP_F32;
    s.early = step_early(e);
    s.bias = y.qk_b;
    s.rope = y.rope;
    s.query = e->lat_query;
    s.cache = r.cache;
    s.gate = e->lat_gate;
    return s;
}
static MambaScanArgs mamba_scan_args(const lpp_engine* e, const ModelLayer& y, const LayerRun& r) {
    MambaScanArgs a = {};
    a.inner = y.d.inner;
    a.state = y.d.state;
    a.dt_rank = y.d.dt_rank;
    a.state_pitch = y.state_pitch;
    a.dt_pitch = y.dt_pitch;
    a.low_rows = y.low_rows;
    a.low = e->scan_low;
    a.w_dt = y.w_dt;
    a.dt_b = y.dt_b;
    a.A = y.A;
    a.D = y.skip;
    a.S = r.S;
    a.x = e->scan_x;
    a.z = e->scan_z;
    a.out = e->att_out;
    a.st = e->st;
    a.seq_len = e->c.seq_len;
    a.early = step_early(e);
    a.taps = y.d.conv;
    a.ring = r.ring;
    a.ring_pitch = y.inner_rows;
    return a;
}
// Limits of a selective-scan layer (registers and shared memory of the scan kernels); lanes per channel and pieces of four
// state elements per lane by the state's size, and with them the elements a channel has in memory.
constexpr int kScanMaxState = 4 * 32 * 8, kScanMaxTaps = 64, kScanMaxRank = 1536;
static int scan_state_pitch(int n) { return n <= 16 ? 16 : n <= 32 ? 32 : n <= 64 ? 64 : n <= 128 ? 128 : n <= 256 ? 256 : kScanMaxState; }
#define LPP_SCAN_DISPATCH(n, F)         \
    do {                                \
        if ((n) <= 16) return F(4, 1);  \
        if ((n) <= 32) return F(4, 2);  \
        if ((n) <= 64) return F(8, 2);  \
        if ((n) <= 128) return F(16, 2);\
        if ((n) <= 256) return F(32, 2);\
        return F(32, 8);                \
    } while (0)
template <typename WT>
static cudaError_t launch_mamba_step(const MambaScanArgs& a, bool pdl, cudaStream_t s) {
    const size_t smem = (size_t)(a.dt_pitch + 2 * a.state_pitch) * 4;
#define LPP_SCAN(L_, NS_)                                                                                                      \
    launch_kernel(mamba_step_kernel<WT, L_, NS_>, dim3((a.inner + kScanStepThreads / L_ - 1) / (kScanStepThreads / L_)), \
                  dim3(kScanStepThreads), smem, s, pdl, a)
    LPP_SCAN_DISPATCH(a.state_pitch, LPP_SCAN);
#undef LPP_SCAN
}
template <int L, int NS>
static cudaError_t launch_mamba_scan_t(const lpp_engine* e, MambaScanArgs a, cudaStream_t s) {
    a.tile_tokens = kPrefillTokens;
    while (a.tile_tokens > 4 && (size_t)mamba_scan_smem<L>(a.dt_pitch, a.state_pitch, a.tile_tokens) > e->smem_optin) a.tile_tokens /= 2;
    const size_t smem = (size_t)mamba_scan_smem<L>(a.dt_pitch, a.state_pitch, a.tile_tokens);
    const cudaError_t r = cudaFuncSetAttribute(mamba_scan_kernel<L, NS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)e->smem_optin);
    if (r != cudaSuccess) return r;
    return launch_kernel(mamba_scan_kernel<L, NS>, dim3((a.inner + kScanChannels<L> - 1) / kScanChannels<L>), dim3(kScanThreads), smem, s, true, a);
}
static cudaError_t launch_mamba_scan(const lpp_engine* e, const MambaScanArgs& a, cudaStream_t s) {
#define LPP_SCAN(L_, NS_) launch_mamba_scan_t<L_, NS_>(e, a, s)
    LPP_SCAN_DISPATCH(a.state_pitch, LPP_SCAN);
#undef LPP_SCAN
}
static cudaError_t launch_mamba_conv(const MambaConvArgs& a, cudaStream_t s) {
    const dim3 grid((a.inner + 4 * kConvThreads - 1) / (4 * kConvThreads), (a.n_tokens + kConvTokens - 1) / kConvTokens, 2), block(kConvThreads);
    switch (a.taps) {
        case 2: return launch_kernel(mamba_conv_kernel<2>, grid, block, 0, s, true, a);
        case 3: return launch_kernel(mamba_conv_kernel<3>, grid, block, 0, s, true, a);
        case 4: return launch_kernel(mamba_conv_kernel<4>, grid, block, 0, s, true, a);
    }
    const size_t smem = (size_t)(kConvTokens + a.taps - 1) * kConvThreads * sizeof(float4);
    const cudaError_t r = cudaFuncSetAttribute(mamba_conv_kernel<0>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)std::max<size_t>(smem, 49152));
    return r != cudaSuccess ? r : launch_kernel(mamba_conv_kernel<0>, grid, block, smem, s, true, a);
}

// ---- one decode step as a sequence of launches (captured into the graph, or run directly)

struct Recorder {
    lpp_engine* e;
    cudaStream_t s;
    bool prev_kernel = false;  // previous stream item was one of our kernels -> PDL edge allowed
    int kernels = 0;
    bool long_ctx = false;  // record the long-context variant of the step (tensor-core attention kernel)
    cudaError_t err = cudaSuccess;
    std::string where;

    bool pdl() const { return prev_kernel && !(e->c.flags & LPP_FLAG_NO_PDL) && !e->profiling; }
    void mark(int kind) {
        if (!e->profiling) return;
        cudaEvent_t ev;
        cudaEventCreate(&ev);
        if (e->profiling_capture)
            cudaEventRecordWithFlags(ev, s, cudaEventRecordExternal);  // becomes an event-record graph node
        else
            cudaEventRecord(ev, s);
        e->prof_events.push_back(ev);
        e->prof_kinds.push_back(kind);
    }
    void check(cudaError_t r, const char* what) {
        if (r != cudaSuccess && err == cudaSuccess) {
            err = r;
            where = what;
        }
        if (tracing() && (e->c.flags & LPP_FLAG_NO_GRAPH)) {
            TRACE("launched %s #%d -> %s; syncing", what, kernels, cudaGetErrorString(r));
            cudaError_t se = cudaStreamSynchronize(s);
            TRACE("  sync -> %s", cudaGetErrorString(se));
        }
    }
};

// LPP_DEBUG_SKIP=<bitmask of Kind> leaves those kernels out of the step (results become
// meaningless): a timing aid that shows what each kernel kind costs inside the replayed graph.
static unsigned skip_mask() {
    const char* v = aid_env("LPP_DEBUG_SKIP");
    return v ? (unsigned)strtol(v, nullptr, 0) : 0u;
}
// only_kind >= 0 (lpp_profile_kind): every other kind is left out of the recorded sequence.
static bool kind_skipped(const lpp_engine* e, int kind) {
    return (skip_mask() & (1u << kind)) || (e->only_kind >= 0 && kind != e->only_kind);
}

template <typename Args>
static void record_gemv(Recorder& R, int kind, int epi, Args a) {
    lpp_engine* e = R.e;
    if (kind_skipped(e, kind)) return;
    a.st = e->st;
    if (const char* dbg = aid_env("LPP_DEBUG_GEMV")) a.debug = (int)strtol(dbg, nullptr, 0);
    if (aid_env("LPP_GEMV_TRACE")) {
        if (e->gtrace && R.kernels < 256) a.trace = e->gtrace + (size_t)R.kernels * e->num_sms * 8;
    }
    a.vocab = e->c.vocab_size;
    a.seq_len = e->c.seq_len;
    a.norm_eps = e->norm_eps;
    a.norm_n = e->c.dim;
    a.emb_scale = e->emb_scale;
    R.mark(kind);
    R.check(launch_gemv(e, epi, e->c.weight_dtype, a, R.pdl(), R.s), "gemv launch");
    R.mark(-1);
    R.prev_kernel = true;
    R.kernels++;
}

static void record_allreduce(Recorder& R, float* buf, int n) {
    lpp_engine* e = R.e;
    if (kind_skipped(e, kAllReduce)) return;
    R.mark(kAllReduce);
    nccl::result_t r = nccl::AllReduce(buf, buf, (size_t)n, nccl::kFloat32, nccl::kSum, e->comm, R.s);
    if (r != 0 && R.err == cudaSuccess) {
        R.err = cudaErrorUnknown;
        R.where = std::string("ncclAllReduce: ") + nccl::GetErrorString(r);
    }
    R.mark(-1);
    R.prev_kernel = false;
}

static bool tp_peer_path(const lpp_engine* e);
static bool tp_cls_sharded(const lpp_engine* e);
static unsigned int* tp_epoch_word(const lpp_engine* e);

// The fused sampler: exact-order kernel by default, tree kernel when asked for or when the vocabulary
// needs more blocks than can be co-resident.
static cudaError_t launch_sampler(lpp_engine* e, cudaStream_t s, bool pdl, bool end_of_step = false) {
    SampleArgs a = {};
    a.logits = e->logits;
    a.vocab = e->c.vocab_size;
    a.st = e->st;
    a.part_max = e->samp_max;
    a.part_idx = e->samp_idx;
    a.part_sum = e->samp_sum;
    a.counter = e->samp_counter;
    a.r_values = e->r_values;
    a.out_tokens = e->out_tokens;
    a.bump = (end_of_step && tp_peer_path(e)) ? tp_epoch_word(e) : nullptr;
    if (e->exact_sampler) {
        SampleExactArgs ea = {};
        ea.base = a;
        ea.sync = e->ex_sync;
        ea.block_sum = e->ex_block_sum;
        ea.entry_count = e->ex_entry_count;
        ea.entries = e->ex_entries;
        ea.scalars = e->ex_scalars;
        return launch_kernel(sample_exact_kernel, dim3(e->sample_blocks), dim3(kSampleThreads), 0, s, pdl, ea);
    }
    return launch_kernel(sample_kernel, dim3(e->sample_blocks), dim3(kSampleThreads), 0, s, pdl, a);
}

// Start and size of the weight matrix a GEMV kind streams in layer l (this rank's share).
static void matrix_span(const lpp_engine* e, int kind, int l, const void** ptr, size_t* bytes) {
    const size_t D = e->c.dim, esz = e->esz;
    const size_t qkv_rows = e->Dq + 2 * (size_t)e->KVd;
    switch (kind) {
        case kQkv: *bytes = qkv_rows * D * esz; *ptr = (const char*)e->wqkv + l * *bytes; break;
        case kOproj: *bytes = D * e->Dq * esz; *ptr = (const char*)e->wo + l * *bytes; break;
        case kGateUp: *bytes = 2 * (size_t)e->Fl * D * esz; *ptr = (const char*)e->w13 + l * *bytes; break;
        case kDown: *bytes = D * e->Fl * esz; *ptr = (const char*)e->w2 + l * *bytes; break;
        default:
            *bytes = (size_t)e->c.vocab_size * D * esz;
            *ptr = e->wcls;
            if (tp_cls_sharded(e)) {  // this rank's vocabulary rows
                *bytes /= e->c.tp_size;
                if (!e->wcls_shard_only) *ptr = (const char*)e->wcls + (size_t)e->c.tp_rank * *bytes;
            }
            break;
    }
}
// What the GEMV (kind, l) should pull towards L2 for its successor in the step: the next matrix, or
// its first LPP_PF_MB MiB (default 8) when it is larger.  The classifier's successor is the first
// layer's QKV matrix of the next token.
static void set_prefetch(const lpp_engine* e, GemvArgs& a, int kind, int l) {
    int nk, nl = l;
    switch (kind) {
        case kQkv: nk = kOproj; break;
        case kOproj: nk = kGateUp; break;
        case kGateUp: nk = kDown; break;
        case kDown: nk = (l + 1 < e->c.n_layers) ? kQkv : kLmHead; nl = l + 1; break;
        default: nk = kQkv; nl = 0; break;
    }
    if (e->c.tp_size < 2) return;  // one GPU: no measurable effect, so a launch's DRAM traffic stays its matrix once
    size_t cap = 8;
    if (const char* v = aid_env("LPP_PF_MB")) cap = (size_t)std::max(0, atoi(v));
    const void* p;
    size_t bytes;
    matrix_span(e, nk, nl, &p, &bytes);
    bytes = std::min(bytes, cap << 20) & ~(size_t)15;
    a.pf = bytes ? p : nullptr;
    a.pf_bytes = (unsigned int)bytes;
}

// ---- tensor-parallel exchange buffer layout: [epoch word, padded to 256 B][2 * n_layers receive areas],
//      a receive area = [tp][dim] 64-bit {value, flag} words
static size_t tp_header_bytes() { return 1024; }  // epoch word at 0, hint counters (one per exchange) from byte 256
static size_t tp_area_bytes(const lpp_engine* e) { return (size_t)e->c.tp_size * e->c.dim * sizeof(unsigned long long); }
static unsigned long long* tp_area(const lpp_engine* e, int p, int ex) {
    return reinterpret_cast<unsigned long long*>(e->peer_base[p] + tp_header_bytes() + (size_t)ex * tp_area_bytes(e));
}
static unsigned int* tp_epoch_word(const lpp_engine* e) { return reinterpret_cast<unsigned int*>(e->tp_buf); }
static unsigned int* tp_hint(const lpp_engine* e, int p, int ex) { return reinterpret_cast<unsigned int*>(e->peer_base[p] + 256) + ex; }
// The arrival hint spares the receive area the polling of every thread of every CTA; with two ranks that
// polling is light and measured faster (2051 against 2078 us/step on the 8B shape), so the hint is used from
// three ranks on (LPP_TP_HINT=0/1 overrides).
static bool tp_use_hint(const lpp_engine* e) {
    if (2 * e->c.n_layers > 192) return false;
    if (const char* v = aid_env("LPP_TP_HINT")) return atoi(v) != 0;
    return e->c.tp_size > 2;
}
static unsigned int tp_hint_per_step(const lpp_engine* e) {
    const int groups = e->c.dim / kRowsPerGroup;  // the producing GEMVs have dim rows
    return (unsigned int)(e->c.tp_size * std::max(1, std::min(groups, e->num_sms)));
}
// (a single-kind timing run must not take part in exchanges: its producers would have no consumers)
static bool tp_peer_path(const lpp_engine* e) {
    return e->c.tp_size > 1 && e->peer_ready && e->only_kind < 0 &&
           !(e->c.flags & (LPP_FLAG_GEMV_LDG | LPP_FLAG_TP_NCCL));
}
// producer side: exchange `ex` takes the rows of this residual GEMV
static void tp_set_producer(const lpp_engine* e, GemvArgs& a, int ex) {
    const bool use_hint = tp_use_hint(e);
    a.tp_size = e->c.tp_size;
    a.tp_epoch = tp_epoch_word(e);
    for (int p = 0; p < e->c.tp_size; ++p) {
        a.tp_out[p] = tp_area(e, p, ex) + (size_t)e->c.tp_rank * e->c.dim;
        a.tp_hint_out[p] = use_hint ? tp_hint(e, p, ex) : nullptr;
    }
}
// consumer side: this GEMV's input is the sum of the slots of exchange `ex`
static void tp_set_consumer(const lpp_engine* e, GemvArgs& a, int ex, float* x_store) {
    a.tp_size = e->c.tp_size;
    a.tp_epoch = tp_epoch_word(e);
    a.tp_in = tp_area(e, e->c.tp_rank, ex);
    a.tp_hint_in = tp_use_hint(e) ? tp_hint(e, e->c.tp_rank, ex) : nullptr;
    a.tp_wait_cycles = e->h_st->tp_wait_cycles > 0 ? e->h_st->tp_wait_cycles : kTpWaitCycles;
    a.tp_hint_per_step = tp_hint_per_step(e);
    a.x = nullptr;
    a.x_store = x_store;
}

// The classifier is sharded by vocabulary rows when the peers are mapped: every rank computes
// vocab/tp logits and stores them, as flagged words, into every rank's logits area (after the
// exchange areas of the buffer); a small kernel turns the words into the float logits the sampler reads.
static bool tp_cls_sharded(const lpp_engine* e) {
    return e->c.tp_size > 1 && tp_peer_path(e) && e->c.vocab_size % (kRowsPerGroup * e->c.tp_size) == 0 && !aid_env("LPP_TP_FULL_CLS");
}
static unsigned long long* tp_logits_area(const lpp_engine* e, int p) {
    return reinterpret_cast<unsigned long long*>(e->peer_base[p] + tp_header_bytes() + (size_t)2 * e->c.n_layers * tp_area_bytes(e));
}

// words [0, n) = {logit, flag}: waits for the local classifier kernel (so that its CTAs, which this kernel's
// CTAs would otherwise sit beside, are not slowed by polling), then polls until every word, local or from a
// peer, carries this step's flag (bounded) and writes the floats.
static __global__ void __launch_bounds__(256) tp_unpack_logits_kernel(const unsigned long long* words, float* logits, int n,
                                                                    const unsigned int* epoch, StepState* st, long long limit) {
    pdl_launch_dependents();
    pdl_wait();
    const unsigned int flag = *epoch + 1u;
    const int i = (blockIdx.x * 256 + threadIdx.x) * 4;
    if (i >= n) return;
    unsigned long long w[4];
    long long t0 = 0;
    while (true) {
        asm volatile("ld.volatile.global.v2.u64 {%0,%1}, [%2];" : "=l"(w[0]), "=l"(w[1]) : "l"(words + i) : "memory");
        asm volatile("ld.volatile.global.v2.u64 {%0,%1}, [%2];" : "=l"(w[2]), "=l"(w[3]) : "l"(words + i + 2) : "memory");
        bool pending = false;
#pragma unroll
        for (int q = 0; q < 4; ++q) pending |= (i + q < n) && (unsigned int)(w[q] >> 32) != flag;
        if (!pending) break;
        if (t0 == 0) {
            if (status_timed_out(st)) break;
            t0 = clock64();
        } else if (clock64() - t0 > limit) {
            atomicOr(&st->status, kStatusBarrierTimeout);
            break;
        }
        __nanosleep(40);
    }
#pragma unroll
    for (int q = 0; q < 4; ++q)
        if (i + q < n) logits[i + q] = __uint_as_float((unsigned int)w[q]);
}

// Ends a step that has no sampler kernel: bumps the exchange epoch.
static __global__ void tp_bump_kernel(unsigned int* epoch) {
    pdl_wait();
    *epoch = *epoch + 1u;
}

// What the kernels after the mixer need to know about a layer, whichever way its weights are stored.
struct LayerView {
    const void *wo, *w13, *w2;
    const float *norm2_w, *norm2_b;
    const float *o_add, *down_add;  // added with the output and the down projection, nullptr = nothing
    int o_k, ff, ff_k;  // inputs of the output projection; feed-forward width (0 = none), inputs of the down projection
    int act;
};
static LayerView layer_view(const lpp_engine* e, int l) {  // l: layer, or run of one
    if (!e->layers.empty()) {
        const LayerRun& r = e->runs[l];
        const ModelLayer& y = e->layers[r.layer];
        return {y.wo, y.w13, y.w2, y.n2w, y.n2b, r.o_add, r.down_add, y.o_pitch, y.d.ff, y.ff_pitch,
                y.d.act == LPP_ACT_GELU_TANH ? kActGeluTanh : kActSilu};
    }
    const size_t D = e->c.dim, esz = e->esz;
    return {(const char*)e->wo + (size_t)l * D * e->Dq * esz, (const char*)e->w13 + (size_t)l * 2 * e->Fl * D * esz,
            (const char*)e->w2 + (size_t)l * D * e->Fl * esz, e->rms_ffn + (size_t)l * D, nullptr, nullptr, nullptr, e->Dq, e->Fl, e->Fl, kActSilu};
}

// Steps of the recorded order: layers, or their runs.
static int n_runs(const lpp_engine* e) { return e->layers.empty() ? e->c.n_layers : (int)e->runs.size(); }
// The loop's vector that is added before the first run, nullptr = none.
static const float* first_add(const lpp_engine* e) {
    return !e->runs.empty() && e->runs[0].step_row >= 0 ? e->loop_vec + (size_t)e->runs[0].step_row * e->Dp : nullptr;
}

// Grouped-query attention of the reference: fused norm + QKV GEMV + RoPE + KV scatter, split-KV flash decode.
static void record_gqa_mixer(Recorder& R, int l, float* cur) {
    lpp_engine* e = R.e;
    const lpp_config& c = e->c;
    const int D = c.dim, qkv_rows = e->Dq + 2 * e->KVd;
    GemvArgs a = {};
    a.W = (const char*)e->wqkv + (size_t)l * qkv_rows * D * e->esz;
    a.n_rows = qkv_rows;
    a.K = D;
    a.norm_w = e->rms_att + (size_t)l * D;
    if (l == 0) {
        a.emb = e->emb;
        a.x_store = cur;
    } else {
        a.x = cur;
        if (tp_peer_path(e)) tp_set_consumer(e, a, 2 * (l - 1) + 1, cur);  // the previous layer's down exchange
    }
    a.out = e->q;
    a.q_rows = e->Dq;
    a.kv_rows = e->KVd;
    a.head_size = e->hs;
    a.rope = e->rope;
    const size_t lofs = (size_t)l * e->KVHl * c.seq_len * e->hs * e->kvesz;
    a.k_cache = (char*)e->kcache + lofs;
    a.v_cache = (char*)e->vcache + lofs;
    a.kv_is_f32 = c.kv_dtype == LPP_F32;
    // split-KV flash decode
    AttnArgs at = {};
    at.q = e->q;
    at.k_cache = a.k_cache;
    at.v_cache = a.v_cache;
    at.out = e->att_out;
    at.part = e->attn_part;
    at.counters = e->attn_counters;
    at.st = e->st;
    at.seq_len = c.seq_len;
    at.head_size = e->hs;
    at.gqa = e->gqa;
    at.n_splits = e->attn_splits;
    at.n_kv_heads = e->KVHl;
    if (const char* mc = aid_env("LPP_ATTN_CHUNK")) at.min_chunk = atoi(mc);  // timing experiments
    set_prefetch(e, a, kQkv, l);
    record_gemv(R, kQkv, kEpiQkv, a);
    dim3 grid(e->attn_splits, e->KVHl, e->attn_z);
    if (kind_skipped(e, kAttn)) return;
    if (e->gtrace && R.kernels < 256) at.trace = e->gtrace + (size_t)R.kernels * e->num_sms * 8;
    R.mark(kAttn);
    if (attn_mma_supported(e) && !aid_env("LPP_ATTN_CUDA_CORES")) {
        at.n_splits = e->attn_splits_long;
        R.check(launch_attn_mma(e, at, R.pdl(), R.s), "attention (tensor-core) launch");
    } else {
        R.check(c.kv_dtype == LPP_F32 ? launch_attn_t<float>(e, at, grid, R.pdl(), R.s)
                                      : launch_attn_t<__half>(e, at, grid, R.pdl(), R.s),
                "attention launch");
    }
    R.mark(-1);
    R.prev_kernel = true;
    R.kernels++;
}

// The input projection of run l: normed residual stream (the embedding row in the first run) times the layer's input matrix.
static void set_mixer_input(const lpp_engine* e, GemvArgs& a, const ModelLayer& y, int l, float* cur) {
    a.W = y.w_in;
    a.n_rows = y.in_rows;
    a.K = e->Dp;
    a.norm_w = y.n1w;
    a.norm_b = y.n1b;
    if (l == 0) {
        a.emb = e->emb;
        a.emb_add = first_add(e);
        a.x_store = cur;
    } else {
        a.x = cur;
    }
}

template <typename F>
static void record_launch(Recorder& R, int kind, const char* what, F launch) {
    if (kind_skipped(R.e, kind)) return;
    R.mark(kind);
    R.check(launch(R.pdl()), what);
    R.mark(-1);
    R.prev_kernel = true;
    R.kernels++;
}

// Attention whose values are its keys: input GEMV, attention over the window (shared_kv.cuh).
static void record_shared_kv_mixer(Recorder& R, int l, float* cur) {
    lpp_engine* e = R.e;
    const LayerRun& r = e->runs[l];
    const ModelLayer& y = e->layers[r.layer];
    GemvSharedKvArgs a = {};
    a.kv = shared_kv_args(e, y, r);
    set_mixer_input(e, a, y, l, cur);
    record_gemv(R, kQkv, kEpiSharedKvIn, a);
    const LatentPlan p = latent_plan(e, y, 1);
    record_launch(R, kAttn, "shared-row attention launch",
                  [&](bool pdl) { return launch_latent_attn(e, p, latent_attn_args(e, y, r, p), true, pdl, R.s); });
}

// Selective scan: input GEMV with the convolution, GEMV of dt | B | C, scan (mamba.cuh).
static void record_mamba_mixer(Recorder& R, int l, float* cur) {
    lpp_engine* e = R.e;
    const LayerRun& r = e->runs[l];
    const ModelLayer& y = e->layers[r.layer];
    GemvMambaArgs a = {};
    a.mb.inner = y.d.inner;
    a.mb.inner_rows = y.inner_rows;
    a.mb.taps = y.d.conv;
    a.mb.early = step_early(e);
    a.mb.conv_w = y.conv_w;
    a.mb.conv_b = y.conv_b;
    a.mb.ring = r.ring;
    a.mb.x = e->scan_x;
    a.mb.z = e->scan_z;
    set_mixer_input(e, a, y, l, cur);
    record_gemv(R, kQkv, kEpiMambaIn, a);
    GemvArgs g = {};
    g.W = y.w_low;
    g.n_rows = y.low_rows;
    g.K = y.inner_pitch;
    g.x = e->scan_x;
    g.out = e->scan_low;
    record_gemv(R, kScanIn, kEpiStore, g);
    const MambaScanArgs m = mamba_scan_args(e, y, r);
    record_launch(R, kScan, "selective scan launch", [&](bool pdl) {
        return e->c.weight_dtype == LPP_BF16 ? launch_mamba_step<__nv_bfloat16>(m, pdl, R.s) : launch_mamba_step<float>(m, pdl, R.s);
    });
}

// Latent attention: input GEMV, query GEMV, attention over the window, value GEMV (latent.cuh).
static void record_latent_mixer(Recorder& R, int l, float* cur) {
    lpp_engine* e = R.e;
    const LayerRun& r = e->runs[l];
    const ModelLayer& y = e->layers[r.layer];
    GemvLatentArgs a = {};
    a.lat = latent_args(e, y, r);
    set_mixer_input(e, a, y, l, cur);
    record_gemv(R, kQkv, kEpiLatentIn, a);
    GemvLatentArgs q = {};
    q.lat = a.lat;
    q.W = y.w_uk;
    q.n_rows = y.d.heads * y.rank_pitch;
    q.K = y.dim_pitch;
    q.x = e->lat_qplain;
    q.group_pairs = y.rank_pitch / kRowsPerGroup;
    record_gemv(R, kLatQuery, kEpiLatentQuery, q);
    const LatentPlan p = latent_plan(e, y, 1);
    record_launch(R, kAttn, "latent attention launch",
                  [&](bool pdl) { return launch_latent_attn(e, p, latent_attn_args(e, y, r, p), false, pdl, R.s); });
    GemvLatentArgs v = {};
    v.lat = a.lat;
    v.W = y.w_uv;
    v.n_rows = y.d.heads * y.vdim_rows;
    v.K = y.val_pitch;
    v.out = e->att_out;
    v.group_pairs = y.vdim_rows / kRowsPerGroup;
    record_gemv(R, kLatValue, kEpiLatentValue, v);
}

static void record_step(Recorder& R, bool with_sampler) {
    lpp_engine* e = R.e;
    const lpp_config& c = e->c;
    const int D = e->Dp, L = n_runs(e);
    const size_t esz = e->esz;
    const bool tp = c.tp_size > 1;
    const bool peers = tp_peer_path(e);  // fused exchange over peer memory instead of an NCCL all-reduce
    float* cur = e->xa;
    float* oth = e->xb;
    for (int l = 0; l < L; ++l) {
        if (e->layers.empty()) {
            record_gqa_mixer(R, l, cur);
        } else {
            switch (e->layers[e->runs[l].layer].d.mixer) {
                case LPP_MIXER_LATENT: record_latent_mixer(R, l, cur); break;
                case LPP_MIXER_SHARED_KV: record_shared_kv_mixer(R, l, cur); break;
                case LPP_MIXER_MAMBA: record_mamba_mixer(R, l, cur); break;
            }
        }
        const LayerView v = layer_view(e, l);
        {  // o_proj + residual
            GemvArgs a = {};
            a.W = v.wo;
            a.n_rows = (c.dim + 1) & ~1;
            a.K = v.o_k;
            a.x = e->att_out;
            a.resid = (!tp || c.tp_rank == 0) ? cur : nullptr;
            a.out = tp ? oth : cur;
            if (peers) tp_set_producer(e, a, 2 * l);
            a.bias = v.o_add;
            set_prefetch(e, a, kOproj, l);
            record_gemv(R, kOproj, v.o_add ? kEpiResidBias : kEpiResid, a);
            if (tp && !peers) {
                record_allreduce(R, oth, D);
                std::swap(cur, oth);
            }
        }
        if (v.ff == 0) continue;  // a layer without a feed-forward
        {  // fused norm + gate|up GEMV + gated activation
            GemvArgs a = {};
            a.W = v.w13;
            a.n_rows = 2 * v.ff;
            a.K = D;
            a.x = cur;
            if (peers) tp_set_consumer(e, a, 2 * l, cur);
            a.norm_w = v.norm2_w;
            a.norm_b = v.norm2_b;
            a.act = v.act;
            a.out = e->hb;
            set_prefetch(e, a, kGateUp, l);
            record_gemv(R, kGateUp, kEpiSwiglu, a);
        }
        {  // down + residual
            GemvArgs a = {};
            a.W = v.w2;
            a.n_rows = (c.dim + 1) & ~1;
            a.K = v.ff_k;
            a.x = e->hb;
            a.resid = (!tp || c.tp_rank == 0) ? cur : nullptr;
            a.out = tp ? oth : cur;
            if (peers) tp_set_producer(e, a, 2 * l + 1);
            a.bias = v.down_add;
            set_prefetch(e, a, kDown, l);
            record_gemv(R, kDown, v.down_add ? kEpiResidBias : kEpiResid, a);
            if (tp && !peers) {
                record_allreduce(R, oth, D);
                std::swap(cur, oth);
            }
        }
    }
    {  // final norm + classifier
        GemvArgs a = {};
        a.W = e->wcls;
        a.n_rows = e->Vp;
        a.K = D;
        a.x = cur;
        if (peers) tp_set_consumer(e, a, 2 * (L - 1) + 1, cur);
        a.norm_w = e->rms_final;
        a.norm_b = e->final_b;
        a.out = e->logits;
        const bool sharded = tp_cls_sharded(e);
        if (sharded) {
            const int Vl = c.vocab_size / c.tp_size, r0 = c.tp_rank * Vl;
            a.W = e->wcls_shard_only ? (const char*)e->wcls : (const char*)e->wcls + (size_t)r0 * D * esz;
            a.n_rows = Vl;
            for (int p = 0; p < c.tp_size; ++p) a.tp_out[p] = tp_logits_area(e, p) + r0;
        }
        set_prefetch(e, a, kLmHead, 0);
        record_gemv(R, kLmHead, kEpiStore, a);
        if (sharded && !kind_skipped(e, kLmHead)) {
            const int V = c.vocab_size;
            R.check(launch_kernel(tp_unpack_logits_kernel, dim3((V + 1023) / 1024), dim3(256), 0, R.s, R.pdl(),
                                  (const unsigned long long*)tp_logits_area(e, c.tp_rank), e->logits, V,
                                  (const unsigned int*)tp_epoch_word(e), e->st,
                                  (long long)(e->h_st->tp_wait_cycles > 0 ? e->h_st->tp_wait_cycles : kTpWaitCycles)),
                    "logits unpack launch");
            R.prev_kernel = true;
            R.kernels++;
        }
    }
    if (!with_sampler && tp_peer_path(e)) {
        // no sampler in this graph to end the step: a one-thread kernel bumps the exchange epoch
        R.check(launch_kernel(tp_bump_kernel, dim3(1), dim3(1), 0, R.s, R.pdl(), tp_epoch_word(e)), "epoch bump launch");
        R.prev_kernel = true;
    }
    if (with_sampler && !kind_skipped(e, kSampler)) {
        R.mark(kSampler);
        R.check(launch_sampler(e, R.s, R.pdl(), true), "sampler launch");
        R.mark(-1);
        R.prev_kernel = true;
        R.kernels++;
    }
}

static lpp_status capture(lpp_engine* e, bool with_sampler, bool long_ctx, cudaGraphExec_t* out, int* kernels) {
    cudaGraph_t g = nullptr;
    CU(cudaStreamBeginCapture(e->stream, cudaStreamCaptureModeThreadLocal));
    Recorder R{e, e->stream};
    R.long_ctx = long_ctx;
    record_step(R, with_sampler);
    cudaError_t ce = cudaStreamEndCapture(e->stream, &g);
    if (R.err != cudaSuccess) {
        if (g) cudaGraphDestroy(g);
        (void)cudaGetLastError();
        return fail(LPP_ERR_CUDA, "%s: %s", R.where.c_str(), cudaGetErrorString(R.err));
    }
    if (ce != cudaSuccess) return fail(LPP_ERR_CUDA, "cudaStreamEndCapture: %s", cudaGetErrorString(ce));
    cudaError_t ie = cudaGraphInstantiate(out, g, 0);
    cudaGraphDestroy(g);
    if (ie != cudaSuccess) return fail(LPP_ERR_CUDA, "cudaGraphInstantiate: %s", cudaGetErrorString(ie));
    if (kernels) *kernels = R.kernels;
    return LPP_OK;
}

// pos: the position this step runs at (known to the host in every mode); it selects the variant.
static lpp_status run_step(lpp_engine* e, bool with_sampler, int pos) {
    const int v = 0;  // a single graph variant serves every position
    (void)pos;
    if (e->c.flags & LPP_FLAG_NO_GRAPH) {
        Recorder R{e, e->stream};
        R.long_ctx = v == 1;
        record_step(R, with_sampler);
        if (R.err != cudaSuccess) return fail(LPP_ERR_CUDA, "%s: %s", R.where.c_str(), cudaGetErrorString(R.err));
        return LPP_OK;
    }
    CU(cudaGraphLaunch(with_sampler ? e->g_full[v] : e->g_logits[v], e->stream));
    return LPP_OK;
}

// ------------------------------------------------------------------ create / destroy

static bool dpl_supported(int hs) {
    const int d = hs / 8;
    return hs % 8 == 0 && (d == 2 || d == 4 || d == 6 || d == 8 || d == 12 || d == 16);
}

// Makes `device` current if it is a GPU this library runs on.
static lpp_status open_device(int device, cudaDeviceProp* prop) {
    int ndev = 0;
    if (cudaGetDeviceCount(&ndev) != cudaSuccess || ndev == 0) {
        (void)cudaGetLastError();
        return fail(LPP_ERR_NO_DEVICE, "no CUDA device");
    }
    if (device < 0 || device >= ndev) return fail(LPP_ERR_INVALID_ARG, "device %d out of range", device);
    CU(cudaSetDevice(device));
    CU(cudaGetDeviceProperties(prop, device));
    if (prop->major < 10) return fail(LPP_ERR_NO_DEVICE, "device is sm_%d%d; this library is built for sm_100a only", prop->major, prop->minor);
    return LPP_OK;
}

// Buffers every kind of engine has: stream, one step's vectors, sampler scratch, step state.  att_n and hb_n are the
// inputs of the output and of the down projection (the largest ones when layers differ).
static lpp_status alloc_step_buffers(lpp_engine* e, size_t att_n, size_t hb_n) {
    const lpp_config& c = e->c;
    const size_t D = e->Dp;
    CU(cudaStreamCreateWithFlags(&e->stream, cudaStreamNonBlocking));
    CU(cudaEventCreate(&e->ev0));
    CU(cudaEventCreate(&e->ev1));
    CU(cudaMalloc(&e->xa, D * 4));
    CU(cudaMalloc(&e->xb, D * 4));
    CU(cudaMalloc(&e->att_out, att_n * 4));
    CU(cudaMalloc(&e->hb, hb_n * 4));
    CU(cudaMalloc(&e->logits, (size_t)e->Vp * 4));
    // padded inputs stay what they are here: zero
    CU(cudaMemsetAsync(e->xa, 0, D * 4, e->stream));
    CU(cudaMemsetAsync(e->xb, 0, D * 4, e->stream));
    CU(cudaMemsetAsync(e->att_out, 0, att_n * 4, e->stream));
    CU(cudaMemsetAsync(e->hb, 0, hb_n * 4, e->stream));
    CU(cudaMalloc(&e->samp_max, e->sample_blocks * 4));
    CU(cudaMalloc(&e->samp_sum, e->sample_blocks * 4));
    CU(cudaMalloc(&e->samp_idx, e->sample_blocks * 4));
    CU(cudaMalloc(&e->samp_counter, 4));
    CU(cudaMemsetAsync(e->samp_counter, 0, 4, e->stream));
    e->exact_sampler = !(c.flags & LPP_FLAG_FAST_SAMPLER) && e->sample_blocks <= e->num_sms;
    if (e->exact_sampler) {
        CU(cudaMalloc(&e->ex_sync, 2 * sizeof(unsigned int)));
        CU(cudaMemsetAsync(e->ex_sync, 0, 2 * sizeof(unsigned int), e->stream));
        CU(cudaMalloc(&e->ex_block_sum, e->sample_blocks * sizeof(double)));
        CU(cudaMalloc(&e->ex_entry_count, e->sample_blocks * sizeof(int)));
        CU(cudaMalloc(&e->ex_entries, (size_t)e->sample_blocks * kExactMaxEntries * sizeof(ExactEntry)));
        CU(cudaMalloc(&e->ex_scalars, 64 * sizeof(float)));
    }
    e->run_cap = std::max<int>(4096, c.seq_len);
    CU(cudaMalloc(&e->r_values, (size_t)e->run_cap * 4));
    CU(cudaMalloc(&e->out_tokens, (size_t)e->run_cap * 4));
    CU(cudaMalloc(&e->st, sizeof(StepState)));
    CU(cudaMemsetAsync(e->st, 0, sizeof(StepState), e->stream));
    CU(cudaMallocHost(&e->h_st, sizeof(StepState)));
    memset(e->h_st, 0, sizeof(StepState));
    {
        int khz = 0;  // SM clock in kHz = clocks per millisecond
        CU(cudaDeviceGetAttribute(&khz, cudaDevAttrClockRate, c.device));
        e->h_st->wait_cycles = c.wait_ms > 0 ? (long long)c.wait_ms * khz : 0;
        e->h_st->tp_wait_cycles = c.tp_wait_ms > 0 ? (long long)c.tp_wait_ms * khz : 0;
    }
    CU(cudaMallocHost(&e->h_out, 16));
    return LPP_OK;
}

extern "C" lpp_status lpp_engine_create(const lpp_config* cfg, const void* nccl_id, lpp_engine** out) {
    if (!cfg || !out) return fail(LPP_ERR_INVALID_ARG, "null argument");
    *out = nullptr;
    const lpp_config& c = *cfg;
    if (c.dim <= 0 || c.hidden_dim <= 0 || c.n_layers <= 0 || c.n_heads <= 0 || c.n_kv_heads <= 0 ||
        c.vocab_size <= 0 || c.seq_len <= 0)
        return fail(LPP_ERR_INVALID_ARG, "non-positive model dimension");
    if (c.dim % c.n_heads || c.n_heads % c.n_kv_heads)
        return fail(LPP_ERR_INVALID_ARG, "dim %% n_heads or n_heads %% n_kv_heads != 0");
    if (c.weight_dtype != LPP_F16 && c.weight_dtype != LPP_F32) return fail(LPP_ERR_INVALID_ARG, "bad weight_dtype");
    if (c.kv_dtype != LPP_F16 && c.kv_dtype != LPP_F32) return fail(LPP_ERR_INVALID_ARG, "bad kv_dtype");
    if (c.tp_size < 1 || c.tp_rank < 0 || c.tp_rank >= c.tp_size) return fail(LPP_ERR_INVALID_ARG, "bad tp rank/size");
    if (c.n_kv_heads % c.tp_size || c.hidden_dim % c.tp_size)
        return fail(LPP_ERR_INVALID_ARG, "tp_size %d must divide n_kv_heads %d and hidden_dim %d", c.tp_size,
                    c.n_kv_heads, c.hidden_dim);
    const int hs = c.dim / c.n_heads;
    if (!dpl_supported(hs)) return fail(LPP_ERR_INVALID_ARG, "head_size %d unsupported (16,32,48,64,96,128)", hs);
    const int vec = c.weight_dtype == LPP_F16 ? 8 : 4;
    const int Fl = c.hidden_dim / c.tp_size;
    const int Dq = c.dim / c.tp_size;
    if (c.dim % vec || Fl % vec || Dq % vec || (c.vocab_size & 1) || (Fl & 1))
        return fail(LPP_ERR_INVALID_ARG, "dim/hidden/vocab not multiples of the vector width");
    if (c.tp_size > 1 && !nccl_id && !(c.flags & LPP_FLAG_TP_LOCAL))
        return fail(LPP_ERR_INVALID_ARG, "tp_size > 1 needs an nccl id (or LPP_FLAG_TP_LOCAL)");
    if ((c.flags & LPP_FLAG_TP_LOCAL) && c.tp_size > kMaxTp)
        return fail(LPP_ERR_INVALID_ARG, "LPP_FLAG_TP_LOCAL supports at most %d ranks", kMaxTp);

    cudaDeviceProp prop;
    TRY(open_device(c.device, &prop));
    TRACE("create: device %d ok (%s, %d SMs)", c.device, prop.name, prop.multiProcessorCount);
    lpp_engine* e = new lpp_engine();
    e->c = c;
    e->hs = hs;
    e->Hl = c.n_heads / c.tp_size;
    e->KVHl = c.n_kv_heads / c.tp_size;
    e->Dq = Dq;
    e->KVd = e->KVHl * hs;
    e->Fl = Fl;
    e->gqa = c.n_heads / c.n_kv_heads;
    e->esz = c.weight_dtype == LPP_F16 ? 2 : 4;
    e->kvesz = c.kv_dtype == LPP_F16 ? 2 : 4;
    e->num_sms = prop.multiProcessorCount;
    e->smem_optin = prop.sharedMemPerBlockOptin;
    e->attn_gb = (e->gqa % 4 == 0) ? 4 : (e->gqa % 2 == 0 ? 2 : 1);  // query heads per attention CTA
    e->attn_z = e->gqa / e->attn_gb;
    int splits = c.attn_splits > 0 ? c.attn_splits : (2 * e->num_sms + e->KVHl * e->attn_z - 1) / (e->KVHl * e->attn_z);
    e->attn_splits = std::max(1, std::min(splits, 64));
    e->attn_splits_long = std::max(1, std::min(e->attn_splits, e->num_sms / std::max(1, e->KVHl)));
    e->sample_blocks = (c.vocab_size + kSampleChunk - 1) / kSampleChunk;
    if (e->sample_blocks > kSampleMaxBlocks) {
        delete e;
        return fail(LPP_ERR_TOO_LARGE, "vocab_size %d exceeds the sampler's %d", c.vocab_size, kSampleMaxBlocks * kSampleChunk);
    }
    e->got.assign((size_t)LPP_T_COUNT * c.n_layers, 0);
    e->Dp = c.dim;
    e->Vp = c.vocab_size;

    auto bail = [&](lpp_status s) {
        lpp_engine_destroy(e);
        return s;
    };
#define CUB(call)                                                                                              \
    do {                                                                                                       \
        cudaError_t e_ = (call);                                                                               \
        if (e_ != cudaSuccess)                                                                                 \
            return bail(fail(LPP_ERR_CUDA, "%s failed: %s (%s:%d)", #call, cudaGetErrorString(e_), __FILE__, __LINE__)); \
    } while (0)
    {
        const lpp_status st = alloc_step_buffers(e, (size_t)e->Dq, (size_t)e->Fl);
        if (st != LPP_OK) return bail(st);
    }
    const size_t D = c.dim, L = c.n_layers, V = c.vocab_size, S = c.seq_len;
    const size_t esz = e->esz;
    CUB(cudaMalloc(&e->wqkv, L * (e->Dq + 2 * (size_t)e->KVd) * D * esz));
    CUB(cudaMalloc(&e->wo, L * D * e->Dq * esz));
    CUB(cudaMalloc(&e->w13, L * 2 * e->Fl * D * esz));
    CUB(cudaMalloc(&e->w2, L * D * e->Fl * esz));
    CUB(cudaMalloc(&e->emb, V * D * esz));
    CUB(cudaMalloc(&e->rms_att, L * D * 4));
    CUB(cudaMalloc(&e->rms_ffn, L * D * 4));
    CUB(cudaMalloc(&e->rms_final, D * 4));
    const size_t kvbytes = L * e->KVHl * S * hs * e->kvesz;
    CUB(cudaMalloc(&e->kcache, kvbytes));
    CUB(cudaMalloc(&e->vcache, kvbytes));
    CUB(cudaMemsetAsync(e->kcache, 0, kvbytes, e->stream));
    CUB(cudaMemsetAsync(e->vcache, 0, kvbytes, e->stream));
    CUB(cudaMalloc(&e->q, (size_t)e->Dq * 4));
    CUB(cudaMalloc(&e->attn_part, (size_t)e->Hl * e->attn_splits * (hs + 2) * 4));
    CUB(cudaMalloc(&e->attn_counters, (size_t)e->KVHl * e->attn_z * 4));
    CUB(cudaMemsetAsync(e->attn_counters, 0, (size_t)e->KVHl * e->attn_z * 4, e->stream));
    TRACE("create: buffers allocated");
    // rope table with libm, evaluated exactly like the reference loop (src/ops.cpp:36-40)
    {
        const int half = hs / 2;
        std::vector<float> freq(half);
        for (int j = 0; j < half; ++j) {
            const int head_dim = 2 * j;
            freq[j] = 1.0f / powf(c.rope_base, head_dim / (float)hs);
        }
        std::vector<float2> tab((size_t)S * half);
        for (size_t p = 0; p < S; ++p)
            for (int j = 0; j < half; ++j) {
                const float val = (int)p * freq[j];
                tab[p * half + j] = make_float2(cosf(val), sinf(val));
            }
        CUB(cudaMalloc(&e->rope, tab.size() * sizeof(float2)));
        CUB(cudaMemcpy(e->rope, tab.data(), tab.size() * sizeof(float2), cudaMemcpyHostToDevice));
    }

    if (c.tp_size > 1 && !(c.flags & LPP_FLAG_TP_LOCAL)) {
        if (!nccl::load()) return bail(fail(LPP_ERR_NCCL, "cannot load libnccl.so.2: %s", dlerror()));
        nccl::unique_id id;
        memcpy(&id, nccl_id, sizeof id);
        nccl::result_t r = nccl::CommInitRank(&e->comm, c.tp_size, id, c.tp_rank);
        if (r != 0) return bail(fail(LPP_ERR_NCCL, "ncclCommInitRank: %s", nccl::GetErrorString(r)));
    }
    if (c.tp_size > 1 && c.tp_size <= kMaxTp) {
        // receive areas and counters of the peer-memory exchange (used once lpp_tp_connect has mapped the peers)
        // and the logits area of the vocabulary-sharded classifier
        e->tp_buf_bytes = tp_header_bytes() + (size_t)2 * c.n_layers * tp_area_bytes(e) +
                          (size_t)c.vocab_size * sizeof(unsigned long long);
        CUB(cudaMalloc(&e->tp_buf, e->tp_buf_bytes));
        CUB(cudaMemset(e->tp_buf, 0, e->tp_buf_bytes));
        e->peer_base[c.tp_rank] = e->tp_buf;
    }
    CUB(cudaStreamSynchronize(e->stream));
#undef CUB
    TRACE("create: done");
    *out = e;
    return LPP_OK;
}

// ------------------------------------------------------------------ engines described layer by layer

// cos / sin of every position and rotated pair.  Frequencies and angles in double, so a far position's angle is as exact as
// a near one's; pairs beyond rot_dims do not turn.  Layers with the same rotation share a table.
static lpp_status rope_table(lpp_engine* e, const lpp_layer_desc& d, const float2** out) {
    *out = nullptr;
    if (d.rot_dim == 0) return LPP_OK;
    for (auto& t : e->rope_tables) {
        const lpp_layer_desc& o = t.first;
        if (o.rot_dim == d.rot_dim && o.rot_dims == d.rot_dims && o.rot_base == d.rot_base && o.yarn_factor == d.yarn_factor &&
            o.yarn_original == d.yarn_original && o.yarn_fast == d.yarn_fast && o.yarn_slow == d.yarn_slow) {
            *out = t.second;
            return LPP_OK;
        }
    }
    const int half = d.rot_dim / 2, S = e->c.seq_len;
    std::vector<double> f(half, 0.0);
    double mag = 1.0;
    for (int i = 0; i < d.rot_dims / 2; ++i) f[i] = pow(d.rot_base, -2.0 * i / d.rot_dims);
    if (d.yarn_factor != 0.0) {
        // the pair whose wave makes `turns` turns over the original context, as a (fractional) dimension index
        auto border = [&](double turns) {
            return d.rot_dims * log(d.yarn_original / (2.0 * M_PI * turns)) / (2.0 * log(d.rot_base));
        };
        const double lo = std::max(floor(border(d.yarn_fast)), 0.0), hi = std::min(ceil(border(d.yarn_slow)), (double)d.rot_dims - 1.0);
        for (int i = 0; i < d.rot_dims / 2; ++i) {
            const double ramp = std::min(std::max((i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
            f[i] = f[i] / d.yarn_factor * ramp + f[i] * (1.0 - ramp);
        }
        mag = 0.1 * log(d.yarn_factor) + 1.0;
    }
    std::vector<float2> tab((size_t)S * half, make_float2(1.f, 0.f));
    for (size_t p = 0; p < (size_t)S; ++p)
        for (int i = 0; i < d.rot_dims / 2; ++i)
            tab[p * half + i] = make_float2((float)(mag * cos((double)p * f[i])), (float)(mag * sin((double)p * f[i])));
    float2* dev = nullptr;
    CU(cudaMalloc(&dev, tab.size() * sizeof(float2)));
    e->rope_tables.push_back({d, dev});
    CU(cudaMemcpy(dev, tab.data(), tab.size() * sizeof(float2), cudaMemcpyHostToDevice));
    *out = dev;
    return LPP_OK;
}

static lpp_status zeroed(lpp_engine* e, void** p, size_t bytes) {
    bytes = std::max<size_t>(bytes, 16);
    CU(cudaMalloc(p, bytes));
    CU(cudaMemsetAsync(*p, 0, bytes, e->stream));
    return LPP_OK;
}
template <typename T>
static lpp_status zeroed(lpp_engine* e, T** p, size_t bytes) {
    return zeroed(e, reinterpret_cast<void**>(p), bytes);
}

static bool layer_has_loop(const lpp_model_desc* m) { return m->loop_times > 0 && m->loop_stop > m->loop_start; }

static lpp_status check_layer(const lpp_layer_desc& d, int l) {
    if (d.ff < 0 || d.window < 0 || d.rot_dims < 0) return fail(LPP_ERR_INVALID_ARG, "layer %d: bad size", l);
    if (d.act != LPP_ACT_SILU && d.act != LPP_ACT_GELU_TANH) return fail(LPP_ERR_INVALID_ARG, "layer %d: unknown activation %d", l, d.act);
    int turnable = 0;  // dimensions of a row that can turn, columns of a cache row's value part
    int cols = 0;
    switch (d.mixer) {
        case LPP_MIXER_LATENT:
            if (d.heads <= 0 || d.dim <= 0 || d.rot_dim < 0 || d.vdim <= 0 || d.kv_rank <= 0) return fail(LPP_ERR_INVALID_ARG, "layer %d: bad size", l);
            turnable = d.rot_dim;
            cols = d.kv_rank;
            break;
        case LPP_MIXER_SHARED_KV:
            if (d.heads <= 0 || d.kv_heads <= 0 || d.heads % d.kv_heads || d.dim <= 0 || !(d.softcap >= 0.f))
                return fail(LPP_ERR_INVALID_ARG, "layer %d: bad size", l);
            turnable = cols = d.dim;
            break;
        case LPP_MIXER_MAMBA:
            if (d.inner <= 0 || d.state <= 0 || d.conv <= 0 || d.dt_rank <= 0) return fail(LPP_ERR_INVALID_ARG, "layer %d: bad size", l);
            if (d.state > kScanMaxState || d.conv > kScanMaxTaps || d.dt_rank > kScanMaxRank)
                return fail(LPP_ERR_TOO_LARGE, "layer %d: state %d, convolution %d or step rank %d", l, d.state, d.conv, d.dt_rank);
            return LPP_OK;
        default: return fail(LPP_ERR_INVALID_ARG, "layer %d: unknown mixer %d", l, d.mixer);
    }
    if (d.rot_dims % 2 || (d.mixer == LPP_MIXER_LATENT && d.rot_dim % 2) || d.rot_dims > turnable) return fail(LPP_ERR_INVALID_ARG, "layer %d: rotation of %d of %d dimensions", l, d.rot_dims, turnable);
    if (d.rot_dims > 0 && !(d.rot_base > 0.0)) return fail(LPP_ERR_INVALID_ARG, "layer %d: bad rotation base", l);
    if (d.yarn_factor != 0.0 && !(d.yarn_factor > 0.0 && d.yarn_original > 0.0 && d.yarn_fast > 0.0 && d.yarn_slow > 0.0))
        return fail(LPP_ERR_INVALID_ARG, "layer %d: bad rotation scaling", l);
    if (cols > kLatentMaxPerThread * kLatentThreads) return fail(LPP_ERR_TOO_LARGE, "layer %d: %d value columns", l, cols);
    return LPP_OK;
}

// The engine's sizes of a layer from its description.
static void size_layer(ModelLayer& y) {
    lpp_layer_desc& d = y.d;
    y.ff_pitch = (int)align_up(d.ff, 64);
    if (d.mixer == LPP_MIXER_MAMBA) {
        y.inner_rows = (int)align_up(d.inner, 4);
        y.inner_pitch = (int)align_up(d.inner, 64);
        y.low_rows = (int)align_up((size_t)d.dt_rank + 2 * d.state, 2);
        y.dt_pitch = (int)align_up(d.dt_rank, 8);
        y.state_pitch = scan_state_pitch(d.state);
        y.in_rows = 2 * y.inner_rows;
        y.o_in = d.inner;
    } else if (d.mixer == LPP_MIXER_SHARED_KV) {
        d.rot_dim = d.rot_dims;  // only what turns has a column of its own
        y.group_heads = d.heads / d.kv_heads;
        y.groups = d.kv_heads;
        y.rank_pitch = (int)align_up(d.dim, 16);
        y.row_width = y.rank_pitch + (int)align_up(d.rot_dim, 16);
        y.head_rows = (int)align_up(d.dim, 2);
        y.q_rows = d.heads * y.head_rows;
        y.k_rows = d.kv_heads * y.head_rows;
        y.in_rows = y.q_rows + y.k_rows + (d.gate ? y.q_rows : 0);
        y.o_in = d.heads * d.dim;
    } else {
        y.group_heads = d.heads;
        y.groups = 1;
        y.rank_pitch = (int)align_up(d.kv_rank, 16);
        y.row_width = y.rank_pitch + (int)align_up(d.rot_dim, 16);
        y.dim_pitch = (int)align_up(d.dim, 64);
        y.val_pitch = (int)align_up(d.kv_rank, 64);
        y.vdim_rows = (int)align_up(d.vdim, 2);
        y.q_plain_rows = (int)align_up((size_t)d.heads * d.dim, 2);
        y.q_rot_rows = d.heads * d.rot_dim;
        y.latent_rows = (int)align_up(d.kv_rank, 2);
        y.in_rows = y.q_plain_rows + y.q_rot_rows + y.latent_rows + d.rot_dim + (int)align_up(d.heads, 2);
        y.o_in = d.heads * d.vdim;
    }
    y.o_pitch = (int)align_up(y.o_in, 64);
}

static lpp_status setup_layer(lpp_engine* e, ModelLayer& y) {
    const lpp_layer_desc& d = y.d;
    const size_t D2 = align_up(e->c.dim, 2), Dp = e->Dp, esz = e->esz;
    TRY(zeroed(e, &y.w_in, (size_t)y.in_rows * Dp * esz));
    TRY(zeroed(e, &y.wo, D2 * y.o_pitch * esz));
    TRY(zeroed(e, &y.n1w, Dp * 4));
    if (e->layer_norm) TRY(zeroed(e, &y.n1b, Dp * 4));
    if (d.ff > 0) {
        TRY(zeroed(e, &y.w13, (size_t)2 * d.ff * Dp * esz));
        TRY(zeroed(e, &y.w2, D2 * y.ff_pitch * esz));
        TRY(zeroed(e, &y.n2w, Dp * 4));
        if (e->layer_norm) TRY(zeroed(e, &y.n2b, Dp * 4));
    }
    if (d.mixer == LPP_MIXER_MAMBA) {
        TRY(zeroed(e, &y.w_low, (size_t)y.low_rows * y.inner_pitch * esz));
        TRY(zeroed(e, &y.w_dt, (size_t)d.inner * y.dt_pitch * esz));
        TRY(zeroed(e, &y.conv_w, (size_t)d.conv * y.inner_rows * 4));
        TRY(zeroed(e, &y.conv_b, (size_t)y.inner_rows * 4));
        TRY(zeroed(e, &y.dt_b, (size_t)d.inner * 4));
        TRY(zeroed(e, &y.A, (size_t)d.inner * y.state_pitch * 4));
        TRY(zeroed(e, &y.skip, (size_t)d.inner * 4));
        return LPP_OK;
    }
    if (d.mixer == LPP_MIXER_LATENT) {
        TRY(zeroed(e, &y.w_uk, (size_t)d.heads * y.rank_pitch * y.dim_pitch * esz));
        TRY(zeroed(e, &y.w_uv, (size_t)d.heads * y.vdim_rows * y.val_pitch * esz));
        TRY(zeroed(e, &y.lat_w, (size_t)y.rank_pitch * 4));
    } else {
        TRY(zeroed(e, &y.qk_b, (size_t)(y.q_rows + y.k_rows) * 4));
        if (d.bias) TRY(zeroed(e, &y.o_b, Dp * 4));
    }
    return rope_table(e, d, &y.rope);
}
static lpp_status setup_run(lpp_engine* e, LayerRun& r) {
    const ModelLayer& y = e->layers[r.layer];
    if (y.d.mixer == LPP_MIXER_MAMBA) {
        TRY(zeroed(e, &r.ring, (size_t)(y.d.conv - 1) * y.inner_rows * 4));
        return zeroed(e, &r.S, (size_t)y.d.inner * y.state_pitch * 4);
    }
    return zeroed(e, &r.cache, (size_t)y.groups * e->c.seq_len * y.row_width * e->kvesz);
}

// What every run adds to the residual stream besides its products: the output's bias, and before a pass of the loop the
// loop's vector, which the run before it adds with its last product.
static lpp_status set_run_adds(lpp_engine* e) {
    for (size_t i = 0; i < e->runs.size(); ++i) {
        LayerRun& r = e->runs[i];
        const ModelLayer& y = e->layers[r.layer];
        const int row = i + 1 < e->runs.size() ? e->runs[i + 1].step_row : -1;
        const float* next = row >= 0 ? e->loop_vec + (size_t)row * e->Dp : nullptr;
        r.o_add = y.o_b;
        r.down_add = nullptr;
        if (!next) continue;
        if (y.d.ff > 0) {
            r.down_add = next;
        } else if (!y.o_b) {
            r.o_add = next;
        } else {
            if (!r.sum_add) TRY(zeroed(e, &r.sum_add, (size_t)e->Dp * 4));
            residual_add_kernel<<<(e->Dp + 255) / 256, 256, 0, e->stream>>>(r.sum_add, y.o_b, next, e->Dp);
            CU(cudaGetLastError());
            r.o_add = r.sum_add;
        }
    }
    return LPP_OK;
}

extern "C" lpp_status lpp_engine_create_layers(const lpp_model_desc* m, const lpp_layer_desc* layers, lpp_engine** out) {
    if (!m || !layers || !out) return fail(LPP_ERR_INVALID_ARG, "null argument");
    *out = nullptr;
    if (m->dim <= 0 || m->vocab_size <= 0 || m->seq_len <= 0 || m->n_layers <= 0)
        return fail(LPP_ERR_INVALID_ARG, "non-positive model dimension");
    if (!((m->weight_dtype == LPP_BF16 && m->kv_dtype == LPP_F16) || (m->weight_dtype == LPP_F32 && m->kv_dtype == LPP_F32)))
        return fail(LPP_ERR_INVALID_ARG, "weights / cache must be BF16 / F16 or F32 / F32");
    if (m->norm != LPP_NORM_RMS && m->norm != LPP_NORM_LAYER) return fail(LPP_ERR_INVALID_ARG, "unknown norm %d", m->norm);
    if (m->loop_times < 0 || m->loop_start < 0 || m->loop_stop < m->loop_start || m->loop_stop > m->n_layers ||
        (m->loop_times == 0 && m->loop_stop > m->loop_start))
        return fail(LPP_ERR_INVALID_ARG, "layers %d .. %d, %d times: not a loop of %d layers", m->loop_start, m->loop_stop, m->loop_times, m->n_layers);
    for (int l = 0; l < m->n_layers; ++l) TRY(check_layer(layers[l], l));
    cudaDeviceProp prop;
    TRY(open_device(m->device, &prop));
    lpp_engine* e = new lpp_engine();
    lpp_config& c = e->c;
    c = {};
    c.dim = m->dim;
    c.n_layers = m->n_layers;
    c.vocab_size = m->vocab_size;
    c.seq_len = m->seq_len;
    c.weight_dtype = m->weight_dtype;
    c.kv_dtype = m->kv_dtype;
    c.tp_size = 1;
    c.device = m->device;
    c.flags = m->flags;
    c.ring_kb = m->ring_kb;
    c.wait_ms = m->wait_ms;
    e->esz = c.weight_dtype == LPP_BF16 ? 2 : 4;
    e->kvesz = c.kv_dtype == LPP_F16 ? 2 : 4;
    e->num_sms = prop.multiProcessorCount;
    e->smem_optin = prop.sharedMemPerBlockOptin;
    e->Dp = (int)align_up(c.dim, 64);
    e->Vp = (int)align_up(c.vocab_size, 2);
    e->layer_norm = m->norm == LPP_NORM_LAYER;
    e->norm_eps = m->norm_eps;
    e->emb_scale = m->emb_scale;
    e->logit_scale = m->logit_scale;
    e->sample_blocks = (c.vocab_size + kSampleChunk - 1) / kSampleChunk;
    e->got.assign((size_t)LPP_T_COUNT * c.n_layers, 0);
    auto bail = [&](lpp_status s) {
        lpp_engine_destroy(e);
        return s;
    };
    if (e->sample_blocks > kSampleMaxBlocks)
        return bail(fail(LPP_ERR_TOO_LARGE, "vocab_size %d exceeds the sampler's %d", c.vocab_size, kSampleMaxBlocks * kSampleChunk));
    // order of execution: the layers before the loop, its passes, the rest
    const bool loop = layer_has_loop(m);
    for (int l = 0; l < (loop ? m->loop_start : c.n_layers); ++l) e->runs.push_back({l});
    if (loop) {
        for (int t = 0; t < m->loop_times; ++t)
            for (int l = m->loop_start; l < m->loop_stop; ++l) e->runs.push_back({l, l == m->loop_start ? t : -1});
        for (int l = m->loop_stop; l < c.n_layers; ++l) e->runs.push_back({l});
    }
    e->layers.resize(c.n_layers);
    size_t att_n = 64, hb_n = 64, qplain_n = 0, raw_n = 0, gate_n = 0, query_n = 0, part_n = 0, heads_n = 0, scan_n = 0, low_n = 0;
    for (int l = 0; l < c.n_layers; ++l) {
        ModelLayer& y = e->layers[l];
        const lpp_layer_desc& d = y.d;
        y.d = layers[l];
        size_layer(y);
        att_n = std::max(att_n, (size_t)y.o_pitch);
        hb_n = std::max(hb_n, (size_t)y.ff_pitch);
        if (d.mixer == LPP_MIXER_MAMBA) {
            e->recurrent = true;
            scan_n = std::max(scan_n, (size_t)y.inner_pitch);
            low_n = std::max(low_n, (size_t)y.low_rows);
            continue;
        }
        query_n = std::max(query_n, (size_t)d.heads * y.row_width);
        part_n = std::max(part_n, (size_t)d.heads * kLatentMaxSplits * (y.rank_pitch + kLatentPartTail));
        heads_n = std::max(heads_n, (size_t)d.heads);
        gate_n = std::max(gate_n, d.mixer == LPP_MIXER_LATENT ? align_up(d.heads, 2) : (size_t)d.heads * d.dim);
        if (d.mixer != LPP_MIXER_LATENT) continue;
        qplain_n = std::max(qplain_n, (size_t)d.heads * y.dim_pitch);
        raw_n = std::max(raw_n, (size_t)y.latent_rows);
    }
    auto setup = [&]() -> lpp_status {
        TRY(alloc_step_buffers(e, att_n, hb_n));
        const size_t Dp = e->Dp;
        TRY(zeroed(e, &e->emb, (size_t)e->Vp * Dp * e->esz));
        TRY(zeroed(e, &e->rms_final, Dp * 4));
        if (e->layer_norm) TRY(zeroed(e, &e->final_b, Dp * 4));
        TRY(zeroed(e, &e->lat_qplain, qplain_n * 4));
        TRY(zeroed(e, &e->lat_raw, raw_n * 4));
        TRY(zeroed(e, &e->lat_gate, gate_n * 4));
        TRY(zeroed(e, &e->lat_query, query_n * e->kvesz));
        TRY(zeroed(e, &e->lat_part, part_n * 4));
        TRY(zeroed(e, &e->row_counters, heads_n * sizeof(unsigned int)));
        TRY(zeroed(e, &e->scan_x, scan_n * 4));
        TRY(zeroed(e, &e->scan_z, scan_n * 4));
        TRY(zeroed(e, &e->scan_low, low_n * 4));
        if (loop) TRY(zeroed(e, &e->loop_vec, (size_t)m->loop_times * Dp * 4));
        e->loop_rows = loop ? m->loop_times : 0;
        for (ModelLayer& y : e->layers) TRY(setup_layer(e, y));
        for (LayerRun& r : e->runs) TRY(setup_run(e, r));
        CU(cudaStreamSynchronize(e->stream));
        return LPP_OK;
    };
    const lpp_status st = setup();
    if (st != LPP_OK) return bail(st);
    *out = e;
    return LPP_OK;
}

extern "C" lpp_status lpp_engine_destroy(lpp_engine* e) {
    if (!e) return LPP_OK;
    cudaSetDevice(e->c.device);
    if (e->stream) cudaStreamSynchronize(e->stream);
    for (int v = 0; v < 2; ++v) {
        if (e->g_full[v]) cudaGraphExecDestroy(e->g_full[v]);
        if (e->g_logits[v]) cudaGraphExecDestroy(e->g_logits[v]);
    }
    if (e->comm) nccl::CommDestroy(e->comm);
    for (int p = 0; p < kMaxTp; ++p)
        if (e->peer_base[p] && p != e->c.tp_rank && e->peer_base[p] != e->absent_peer) cudaIpcCloseMemHandle(e->peer_base[p]);
    if (e->absent_peer) cudaFree(e->absent_peer);
    if (e->tp_buf) cudaFree(e->tp_buf);
    void* bufs[] = {e->wqkv, e->wo, e->w13, e->w2, e->emb, e->wcls_owned ? e->wcls : nullptr, e->rms_att, e->rms_ffn,
                    e->rms_final, e->kcache, e->vcache, e->xa, e->xb, e->q, e->att_out, e->hb, e->logits,
                    e->attn_part, e->attn_counters, e->samp_max, e->samp_sum, e->samp_idx, e->samp_counter,
                    e->r_values, e->out_tokens, e->st, e->rope, e->stage, e->gtrace, e->pf_x, e->pf_q, e->pf_part, e->pf_xn, e->pf_att, e->pf_hb,
                    e->pf_tokens, e->ex_sync, e->ex_block_sum, e->ex_entry_count, e->ex_entries, e->ex_scalars, e->final_b, e->lat_qplain,
                    e->lat_raw, e->lat_gate, e->lat_query, e->lat_part, e->pf_rows, e->pf_logits, e->pf_qn, e->pf_olat, e->pf_lq,
                    e->pf_lpart, e->pf_gate, e->loop_vec, e->scan_x, e->scan_z, e->scan_low, e->row_counters, e->pf_sx, e->pf_sz, e->pf_tail, e->pf_sxp, e->pf_low};
    for (void* p : bufs)
        if (p) cudaFree(p);
    for (const ModelLayer& y : e->layers)
        for (void* p : {y.w_in, y.w_uk, y.w_uv, y.wo, y.w13, y.w2, (void*)y.n1w, (void*)y.n1b, (void*)y.n2w, (void*)y.n2b, (void*)y.lat_w, (void*)y.o_b,
                        (void*)y.qk_b, y.w_low, y.w_dt, (void*)y.conv_w, (void*)y.conv_b, (void*)y.dt_b, (void*)y.A, (void*)y.skip})
            if (p) cudaFree(p);
    for (const LayerRun& r : e->runs)
        for (void* p : {r.cache, (void*)r.ring, (void*)r.S, (void*)r.sum_add})
            if (p) cudaFree(p);
    for (auto& t : e->rope_tables) cudaFree(t.second);
    if (e->h_st) cudaFreeHost(e->h_st);
    if (e->h_out) cudaFreeHost(e->h_out);
    if (e->ev0) cudaEventDestroy(e->ev0);
    if (e->ev1) cudaEventDestroy(e->ev1);
    if (e->stream) cudaStreamDestroy(e->stream);
    delete e;
    return LPP_OK;
}

extern "C" lpp_status lpp_nccl_unique_id(void* out128) {
    if (!out128) return fail(LPP_ERR_INVALID_ARG, "null argument");
    if (!nccl::load()) return fail(LPP_ERR_NCCL, "cannot load libnccl.so.2: %s", dlerror());
    nccl::unique_id id;
    nccl::result_t r = nccl::GetUniqueId(&id);
    if (r != 0) return fail(LPP_ERR_NCCL, "ncclGetUniqueId: %s", nccl::GetErrorString(r));
    memcpy(out128, &id, sizeof id);
    return LPP_OK;
}

// ------------------------------------------------------------------ weight upload

static lpp_status ensure_stage(lpp_engine* e, size_t bytes) {
    if (bytes <= e->stage_bytes) return LPP_OK;
    if (e->stage) CU(cudaFree(e->stage));
    e->stage = nullptr;
    e->stage_bytes = 0;
    CU(cudaMalloc(&e->stage, bytes));
    e->stage_bytes = bytes;
    return LPP_OK;
}

// Element (r, c) of a block of rows x cols: source row r sits at src + ((r / group) * group_stride + r % group) * src_pitch
// (group 0 = consecutive rows), destination dst + r * dst_row + c * dst_col; strides in elements.
struct BlockShape {
    int rows, cols;
    size_t src_pitch;
    int group = 0;
    size_t group_stride = 0;
    size_t dst_row = 0, dst_col = 1;
};
template <typename DT>
static void launch_repack(DT* dst, const void* src, int src_dtype, const BlockShape& b, cudaStream_t s) {
    const long long total = (long long)b.rows * b.cols;
    const int grid = (int)std::min<long long>((total + 255) / 256, 148 * 16);
    const int group = b.group > 0 ? b.group : std::max(1, b.rows);
    const long long gs = b.group > 0 ? (long long)b.group_stride : b.rows;
    if (src_dtype == LPP_F16)
        repack_kernel<DT, __half><<<grid, 256, 0, s>>>(dst, b.dst_row, b.dst_col, (const __half*)src, b.src_pitch, group, gs, b.rows, b.cols);
    else if (src_dtype == LPP_BF16)
        repack_kernel<DT, __nv_bfloat16><<<grid, 256, 0, s>>>(dst, b.dst_row, b.dst_col, (const __nv_bfloat16*)src, b.src_pitch, group, gs, b.rows, b.cols);
    else
        repack_kernel<DT, float><<<grid, 256, 0, s>>>(dst, b.dst_row, b.dst_col, (const float*)src, b.src_pitch, group, gs, b.rows, b.cols);
}
static size_t dtype_size(int t) { return t == LPP_F32 ? 4 : 2; }
static lpp_status put_shape(lpp_engine* e, void* dst, int dst_dtype, const void* src, int src_dtype, int memkind, BlockShape b) {
    const char* p = (const char*)src;
    const size_t sesz = dtype_size(src_dtype);
    if (memkind == LPP_MEM_HOST) {
        // the rows from the first to the last one, compacted to `cols` columns
        const size_t span = b.group > 0 ? (size_t)((b.rows - 1) / b.group) * b.group_stride + (b.rows - 1) % b.group + 1 : b.rows;
        TRY(ensure_stage(e, span * b.cols * sesz));
        CU(cudaMemcpy2DAsync(e->stage, (size_t)b.cols * sesz, p, b.src_pitch * sesz, (size_t)b.cols * sesz, span, cudaMemcpyHostToDevice, e->stream));
        p = (const char*)e->stage;
        b.src_pitch = b.cols;
    }
    if (dst_dtype == LPP_F16)
        launch_repack((__half*)dst, p, src_dtype, b, e->stream);
    else if (dst_dtype == LPP_BF16)
        launch_repack((__nv_bfloat16*)dst, p, src_dtype, b, e->stream);
    else
        launch_repack((float*)dst, p, src_dtype, b, e->stream);
    CU(cudaGetLastError());
    // the staging buffer is reused by the next call and host memory may be freed by the caller
    CU(cudaStreamSynchronize(e->stream));
    return LPP_OK;
}

// dst[r*dst_pitch + c] (dst_dtype) = src[(r0 + r)*src_pitch + c0 + c] (src_dtype), r < rows, c < cols
static lpp_status put_block(lpp_engine* e, void* dst, size_t dst_pitch, int dst_dtype, const void* src,
                            size_t src_pitch, size_t r0, size_t c0, int rows, int cols, int src_dtype, int memkind) {
    BlockShape b;
    b.rows = rows;
    b.cols = cols;
    b.src_pitch = src_pitch;
    b.dst_row = dst_pitch;
    return put_shape(e, dst, dst_dtype, (const char*)src + (r0 * src_pitch + c0) * dtype_size(src_dtype), src_dtype, memkind, b);
}

static bool tensor_expected(const lpp_engine* e, int t, int l);
static __global__ void scale_kernel(float* p, int n, float f) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) p[i] *= f;
}
// p <- -exp(p) for a block of rows x cols
static __global__ void neg_exp_kernel(float* p, int rows, int cols, int pitch) {
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long long)rows * cols) return;
    float* v = p + i / cols * pitch + i % cols;
    *v = (float)-exp((double)*v);
}

// A tensor of an engine described layer by layer, into the padded layouts of ModelLayer.
static lpp_status upload_layered(lpp_engine* e, int which, int l, const void* src, int dt, int memkind) {
    const lpp_config& c = e->c;
    ModelLayer& y = e->layers[l];
    const lpp_layer_desc& d = y.d;
    const int D = c.dim, wd = c.weight_dtype;
    const size_t Dp = e->Dp, esz = e->esz;
    auto vec = [&](float* dst, int n) { return put_block(e, dst, n, LPP_F32, src, n, 0, 0, 1, n, dt, memkind); };
    auto mat = [&](void* dst, size_t pitch, int rows, int cols) { return put_block(e, dst, pitch, wd, src, cols, 0, 0, rows, cols, dt, memkind); };
    auto in_row = [&](size_t r) { return (char*)y.w_in + r * Dp * esz; };
    const bool norm_bias = which == LPP_T_NORM1_B || which == LPP_T_NORM2_B || which == LPP_T_NORM_FINAL_B;
    if (norm_bias && !e->layer_norm) return fail(LPP_ERR_INVALID_ARG, "this model's norms have no bias");
    const bool ff = which == LPP_T_RMS_FFN || which == LPP_T_NORM2_B || which == LPP_T_W1 || which == LPP_T_W2 || which == LPP_T_W3;
    if (ff && d.ff == 0) return fail(LPP_ERR_INVALID_ARG, "layer %d has no feed-forward", l);
    if (which != LPP_T_W_CLS && !tensor_expected(e, which, l)) return fail(LPP_ERR_INVALID_ARG, "tensor id %d does not belong to this model", which);
    auto final_vec = [&](float* dst) -> lpp_status {  // logits are linear in the last norm's output: their factor goes into its weights
        TRY(vec(dst, D));
        scale_kernel<<<(D + 255) / 256, 256, 0, e->stream>>>(dst, D, e->logit_scale);
        CU(cudaGetLastError());
        return LPP_OK;
    };
    // rows of heads (dim each) into sections of the input matrix, head_rows apart
    auto heads = [&](size_t r0, int n) -> lpp_status {
        for (int h = 0; h < n; ++h) TRY(put_block(e, in_row(r0 + (size_t)h * y.head_rows), Dp, wd, src, D, (size_t)h * d.dim, 0, d.dim, D, dt, memkind));
        return LPP_OK;
    };
    switch (which) {
        case LPP_T_TOK_EMB: return mat(e->emb, Dp, c.vocab_size, D);
        case LPP_T_W_CLS:
            if (!e->wcls_owned) {
                TRY(zeroed(e, &e->wcls, (size_t)e->Vp * Dp * esz));
                e->wcls_owned = true;
            }
            return mat(e->wcls, Dp, c.vocab_size, D);
        case LPP_T_RMS_FINAL: return final_vec(e->rms_final);
        case LPP_T_NORM_FINAL_B: return final_vec(e->final_b);
        case LPP_T_RMS_ATT: return vec(y.n1w, D);
        case LPP_T_NORM1_B: return vec(y.n1b, D);
        case LPP_T_RMS_FFN: return vec(y.n2w, D);
        case LPP_T_NORM2_B: return vec(y.n2b, D);
        case LPP_T_LAT_NORM: return vec(y.lat_w, d.kv_rank);
        case LPP_T_LAT_Q: {  // per head dim plain rows, then rot rows: two sections of the input matrix
            BlockShape b;
            b.cols = D;
            b.src_pitch = D;
            b.group_stride = d.dim + d.rot_dim;
            b.dst_row = Dp;
            b.rows = d.heads * d.dim;
            b.group = d.dim;
            TRY(put_shape(e, in_row(0), wd, src, dt, memkind, b));
            if (d.rot_dim == 0) return LPP_OK;
            b.rows = d.heads * d.rot_dim;
            b.group = d.rot_dim;
            return put_shape(e, in_row(y.q_plain_rows), wd, (const char*)src + (size_t)d.dim * D * dtype_size(dt), dt, memkind, b);
        }
        case LPP_T_LAT_DKV: {  // the latent's section may end in a padding row
            const size_t r0 = (size_t)y.q_plain_rows + y.q_rot_rows;
            TRY(put_block(e, in_row(r0), Dp, wd, src, D, 0, 0, d.kv_rank, D, dt, memkind));
            if (d.rot_dim == 0) return LPP_OK;
            return put_block(e, in_row(r0 + y.latent_rows), Dp, wd, src, D, d.kv_rank, 0, d.rot_dim, D, dt, memkind);
        }
        case LPP_T_LAT_G: return mat(in_row((size_t)y.q_plain_rows + y.q_rot_rows + y.latent_rows + d.rot_dim), Dp, d.heads, D);
        case LPP_T_LAT_UK:  // [heads][dim][rank] -> [heads][rank_pitch][dim_pitch]: the step multiplies by the transpose
            for (int h = 0; h < d.heads; ++h) {
                BlockShape b;
                b.rows = d.dim;
                b.cols = d.kv_rank;
                b.src_pitch = d.kv_rank;
                b.dst_row = 1;
                b.dst_col = y.dim_pitch;
                TRY(put_shape(e, (char*)y.w_uk + (size_t)h * y.rank_pitch * y.dim_pitch * esz, wd,
                              (const char*)src + (size_t)h * d.dim * d.kv_rank * dtype_size(dt), dt, memkind, b));
            }
            return LPP_OK;
        case LPP_T_LAT_UV:
            for (int h = 0; h < d.heads; ++h)
                TRY(put_block(e, (char*)y.w_uv + (size_t)h * y.vdim_rows * y.val_pitch * esz, y.val_pitch, wd, src, d.kv_rank,
                              (size_t)h * d.vdim, 0, d.vdim, d.kv_rank, dt, memkind));
            return LPP_OK;
        case LPP_T_WO: return mat(y.wo, y.o_pitch, D, y.o_in);
        case LPP_T_LOOP_STEP: return put_block(e, e->loop_vec, Dp, LPP_F32, src, D, 0, 0, e->loop_rows, D, dt, memkind);
        case LPP_T_WQ: return heads(0, d.heads);
        case LPP_T_WK: return heads(y.q_rows, d.kv_heads);
        case LPP_T_WG: return heads((size_t)y.q_rows + y.k_rows, d.heads);
        case LPP_T_WQ_B: return put_block(e, y.qk_b, y.head_rows, LPP_F32, src, d.dim, 0, 0, d.heads, d.dim, dt, memkind);
        case LPP_T_WK_B: return put_block(e, y.qk_b + y.q_rows, y.head_rows, LPP_F32, src, d.dim, 0, 0, d.kv_heads, d.dim, dt, memkind);
        case LPP_T_WO_B: return vec(y.o_b, D);
        case LPP_T_SCAN_IN:
            TRY(put_block(e, y.w_in, Dp, wd, src, D, 0, 0, d.inner, D, dt, memkind));
            return put_block(e, in_row(y.inner_rows), Dp, wd, src, D, d.inner, 0, d.inner, D, dt, memkind);
        case LPP_T_SCAN_CONV: {  // [inner][taps] -> [taps][inner_rows]
            BlockShape b;
            b.rows = d.inner;
            b.cols = d.conv;
            b.src_pitch = d.conv;
            b.dst_row = 1;
            b.dst_col = y.inner_rows;
            return put_shape(e, y.conv_w, LPP_F32, src, dt, memkind, b);
        }
        case LPP_T_SCAN_CONV_B: return vec(y.conv_b, d.inner);
        case LPP_T_SCAN_LOW: return mat(y.w_low, y.inner_pitch, d.dt_rank + 2 * d.state, d.inner);
        case LPP_T_SCAN_DT: return mat(y.w_dt, y.dt_pitch, d.inner, d.dt_rank);
        case LPP_T_SCAN_DT_B: return vec(y.dt_b, d.inner);
        case LPP_T_SCAN_D: return vec(y.skip, d.inner);
        case LPP_T_SCAN_A_LOG: {
            TRY(put_block(e, y.A, y.state_pitch, LPP_F32, src, d.state, 0, 0, d.inner, d.state, dt, memkind));
            const long long n = (long long)d.inner * d.state;
            neg_exp_kernel<<<(unsigned int)((n + 255) / 256), 256, 0, e->stream>>>(y.A, d.inner, d.state, y.state_pitch);
            CU(cudaGetLastError());
            return LPP_OK;
        }
        case LPP_T_W1: return put_block(e, y.w13, 2 * Dp, wd, src, D, 0, 0, d.ff, D, dt, memkind);                      // gate -> even rows
        case LPP_T_W3: return put_block(e, (char*)y.w13 + Dp * esz, 2 * Dp, wd, src, D, 0, 0, d.ff, D, dt, memkind);  // up -> odd rows
        case LPP_T_W2: return mat(y.w2, y.ff_pitch, D, d.ff);
    }
    return fail(LPP_ERR_INVALID_ARG, "tensor id %d does not belong to this model", which);
}
// Whether layer l of the model has tensor t.
static bool tensor_expected(const lpp_engine* e, int t, int l) {
    if (t == LPP_T_W_CLS) return false;  // optional
    if (e->layers.empty()) return t < LPP_T_NORM1_B;
    const lpp_layer_desc& d = e->layers[l].d;
    switch (t) {
        case LPP_T_TOK_EMB: case LPP_T_RMS_FINAL: case LPP_T_RMS_ATT: case LPP_T_WO: return true;
        case LPP_T_NORM1_B: case LPP_T_NORM_FINAL_B: return e->layer_norm;
        case LPP_T_NORM2_B: return e->layer_norm && d.ff > 0;
        case LPP_T_RMS_FFN: case LPP_T_W1: case LPP_T_W2: case LPP_T_W3: return d.ff > 0;
        case LPP_T_LOOP_STEP: return e->loop_rows > 0;
        case LPP_T_LAT_Q: case LPP_T_LAT_DKV: case LPP_T_LAT_NORM: case LPP_T_LAT_UK: case LPP_T_LAT_UV: case LPP_T_LAT_G:
            return d.mixer == LPP_MIXER_LATENT;
        case LPP_T_WQ: case LPP_T_WK: return d.mixer == LPP_MIXER_SHARED_KV;
        case LPP_T_WQ_B: case LPP_T_WK_B: case LPP_T_WO_B: return d.mixer == LPP_MIXER_SHARED_KV && d.bias;
        case LPP_T_WG: return d.mixer == LPP_MIXER_SHARED_KV && d.gate;
        case LPP_T_SCAN_IN: case LPP_T_SCAN_CONV: case LPP_T_SCAN_CONV_B: case LPP_T_SCAN_LOW: case LPP_T_SCAN_DT: case LPP_T_SCAN_DT_B:
        case LPP_T_SCAN_A_LOG: case LPP_T_SCAN_D:
            return d.mixer == LPP_MIXER_MAMBA;
    }
    return false;
}
static bool tensor_stacked(int t) {
    return !(t == LPP_T_TOK_EMB || t == LPP_T_RMS_FINAL || t == LPP_T_W_CLS || t == LPP_T_NORM_FINAL_B || t == LPP_T_LOOP_STEP);
}

extern "C" lpp_status lpp_upload_tensor(lpp_engine* e, int which, int layer, const void* src, int src_dtype,
                                        int memkind) {
    if (!e || !src) return fail(LPP_ERR_INVALID_ARG, "null argument");
    if (which < 0 || which >= LPP_T_COUNT) return fail(LPP_ERR_INVALID_ARG, "unknown tensor id %d", which);
    if (src_dtype != LPP_F16 && src_dtype != LPP_F32 && src_dtype != LPP_BF16) return fail(LPP_ERR_INVALID_ARG, "bad src_dtype");
    if (memkind != LPP_MEM_HOST && memkind != LPP_MEM_DEVICE) return fail(LPP_ERR_INVALID_ARG, "bad memkind");
    const lpp_config& c = e->c;
    const bool stacked = tensor_stacked(which);
    if (stacked && (layer < 0 || layer >= c.n_layers)) return fail(LPP_ERR_INVALID_ARG, "layer %d out of range", layer);
    if (!stacked) layer = 0;
    CU(cudaSetDevice(c.device));
    TRACE("upload tensor %d layer %d", which, layer);
    if (!e->layers.empty()) {
        TRY(upload_layered(e, which, layer, src, src_dtype, memkind));
        e->got[(size_t)which * c.n_layers + layer] = 1;
        e->finalized = false;
        return LPP_OK;
    }
    const size_t D = c.dim, F = c.hidden_dim, V = c.vocab_size, esz = e->esz;
    const size_t l = layer, r = c.tp_rank;
    const size_t qkv_rows = e->Dq + 2 * (size_t)e->KVd;
    const int wd = c.weight_dtype;
    char* wqkv_l = (char*)e->wqkv + l * qkv_rows * D * esz;
    char* w13_l = (char*)e->w13 + l * 2 * e->Fl * D * esz;
    lpp_status s = LPP_OK;
    switch (which) {
        default: return fail(LPP_ERR_INVALID_ARG, "tensor id %d does not belong to this model", which);
        case LPP_T_TOK_EMB:
            s = put_block(e, e->emb, D, wd, src, D, 0, 0, (int)V, (int)D, src_dtype, memkind);
            break;
        case LPP_T_W_CLS:
            // With the peers mapped (lpp_tp_connect comes before the uploads in that case) the classifier is
            // sharded by vocabulary rows and this rank never reads another rank's rows: it keeps V/tp rows.
            if (!e->wcls_owned) {
                e->wcls_shard_only = tp_cls_sharded(e);
                CU(cudaMalloc(&e->wcls, (e->wcls_shard_only ? V / c.tp_size : V) * D * esz));
                e->wcls_owned = true;
            }
            if (e->wcls_shard_only)
                s = put_block(e, e->wcls, D, wd, src, D, r * (V / c.tp_size), 0, (int)(V / c.tp_size), (int)D, src_dtype, memkind);
            else
                s = put_block(e, e->wcls, D, wd, src, D, 0, 0, (int)V, (int)D, src_dtype, memkind);
            break;
        case LPP_T_RMS_ATT:
            s = put_block(e, e->rms_att + l * D, D, LPP_F32, src, D, 0, 0, 1, (int)D, src_dtype, memkind);
            break;
        case LPP_T_RMS_FFN:
            s = put_block(e, e->rms_ffn + l * D, D, LPP_F32, src, D, 0, 0, 1, (int)D, src_dtype, memkind);
            break;
        case LPP_T_RMS_FINAL:
            s = put_block(e, e->rms_final, D, LPP_F32, src, D, 0, 0, 1, (int)D, src_dtype, memkind);
            break;
        case LPP_T_WQ:  // row slice of [D][D]
            s = put_block(e, wqkv_l, D, wd, src, D, r * e->Dq, 0, e->Dq, (int)D, src_dtype, memkind);
            break;
        case LPP_T_WK:  // row slice of [KV][D]
            s = put_block(e, wqkv_l + (size_t)e->Dq * D * esz, D, wd, src, D, r * e->KVd, 0, e->KVd, (int)D, src_dtype, memkind);
            break;
        case LPP_T_WV:
            s = put_block(e, wqkv_l + ((size_t)e->Dq + e->KVd) * D * esz, D, wd, src, D, r * e->KVd, 0, e->KVd, (int)D, src_dtype, memkind);
            break;
        case LPP_T_WO:  // column slice of [D][D] (columns = this rank's heads), repacked contiguous
            s = put_block(e, (char*)e->wo + l * D * e->Dq * esz, e->Dq, wd, src, D, 0, r * e->Dq, (int)D, e->Dq, src_dtype, memkind);
            break;
        case LPP_T_W1:  // gate rows -> even rows of w13
            s = put_block(e, w13_l, 2 * D, wd, src, D, r * e->Fl, 0, e->Fl, (int)D, src_dtype, memkind);
            break;
        case LPP_T_W3:  // up rows -> odd rows of w13
            s = put_block(e, w13_l + D * esz, 2 * D, wd, src, D, r * e->Fl, 0, e->Fl, (int)D, src_dtype, memkind);
            break;
        case LPP_T_W2:  // column slice of [D][F]
            s = put_block(e, (char*)e->w2 + l * D * e->Fl * esz, e->Fl, wd, src, F, 0, r * e->Fl, (int)D, e->Fl, src_dtype, memkind);
            break;
    }
    TRY(s);
    e->got[(size_t)which * c.n_layers + layer] = 1;
    e->finalized = false;
    return LPP_OK;
}

extern "C" lpp_status lpp_finalize(lpp_engine* e) {
    if (!e) return fail(LPP_ERR_INVALID_ARG, "null argument");
    const lpp_config& c = e->c;
    CU(cudaSetDevice(c.device));
    static const char* names[LPP_T_COUNT] = {"tok_emb", "rms_att", "wq", "wk", "wv", "wo", "rms_ffn", "w1", "w2", "w3", "rms_final", "w_cls",
                                              "norm1_b", "norm2_b", "norm_final_b", "lat_q", "lat_dkv", "lat_norm", "lat_uk", "lat_uv", "lat_g", "wq_b", "wk_b", "wo_b", "wg",
                                              "scan_in", "scan_conv", "scan_conv_b", "scan_low", "scan_dt", "scan_dt_b", "scan_a_log", "scan_d", "loop_step"};
    for (int t = 0; t < LPP_T_COUNT; ++t) {
        const int n = tensor_stacked(t) ? c.n_layers : 1;
        for (int l = 0; l < n; ++l)
            if (tensor_expected(e, t, l) && !e->got[(size_t)t * c.n_layers + l])
                return fail(LPP_ERR_NOT_READY, "tensor %s (layer %d) was never uploaded", names[t], l);
    }
    if (c.tp_size > 1 && !e->comm && !tp_peer_path(e))
        return fail(LPP_ERR_NOT_READY, "a tensor-parallel engine without NCCL (LPP_FLAG_TP_LOCAL) needs lpp_tp_connect");
    if (e->wcls_shard_only && !tp_cls_sharded(e))
        return fail(LPP_ERR_NOT_READY, "the classifier was uploaded as a vocabulary shard but the engine no longer shards it");
    if (!e->wcls_owned) e->wcls = e->emb;  // tied classifier (src/loader.cpp:66, 471)
    if (e->stage) {
        cudaFree(e->stage);
        e->stage = nullptr;
        e->stage_bytes = 0;
    }
    TRY(set_run_adds(e));
    e->state_len = e->recurrent ? -1 : 0;
    for (int v = 0; v < 2; ++v) {
        if (e->g_full[v]) cudaGraphExecDestroy(e->g_full[v]), e->g_full[v] = nullptr;
        if (e->g_logits[v]) cudaGraphExecDestroy(e->g_logits[v]), e->g_logits[v] = nullptr;
    }
    TRACE("finalize: weights complete");
    if (aid_env("LPP_GEMV_TRACE") && !e->gtrace) {
        CU(cudaMalloc(&e->gtrace, (size_t)256 * e->num_sms * 8 * sizeof(unsigned long long)));
        CU(cudaMemset(e->gtrace, 0, (size_t)256 * e->num_sms * 8 * sizeof(unsigned long long)));
    }
    if (!(c.flags & LPP_FLAG_NO_GRAPH)) {
        for (int v = 0; v < 1; ++v) {
            TRY(capture(e, true, v == 1, &e->g_full[v], v == 0 ? &e->kernels_full : nullptr));
            TRY(capture(e, false, v == 1, &e->g_logits[v], nullptr));
        }
        TRACE("finalize: graphs captured (%d kernels per long-context step)", e->kernels_full);
    } else {
        e->kernels_full = 2 + (tp_cls_sharded(e) ? 1 : 0);
        for (int l = 0; l < n_runs(e); ++l) {
            const int mixer = e->layers.empty() ? 0 : e->layers[e->runs[l].layer].d.mixer;
            e->kernels_full += (mixer == LPP_MIXER_LATENT ? 4 : mixer == LPP_MIXER_MAMBA ? 3 : 2) + 1 + (layer_view(e, l).ff > 0 ? 2 : 0);
        }
    }
    e->finalized = true;
    return LPP_OK;
}

// ------------------------------------------------------------------ stepping

static lpp_status push_state(lpp_engine* e, int token, int pos, const lpp_sample_params* sp, const int* hist,
                             int hist_len, float r, int advance, int window) {
    const lpp_config& c = e->c;
    if (token < 0 || token >= c.vocab_size) return fail(LPP_ERR_INVALID_ARG, "token %d outside [0, %d)", token, c.vocab_size);
    if (pos < 0 || pos >= c.seq_len) return fail(LPP_ERR_INVALID_ARG, "pos %d outside [0, %d)", pos, c.seq_len);
    if (hist_len < 0 || hist_len > kHistoryMax) return fail(LPP_ERR_TOO_LARGE, "history_len %d > %d", hist_len, kHistoryMax);
    StepState* h = e->h_st;
    h->token = token;
    h->pos = pos;
    const bool use_hist = sp && sp->penalty > 1.0f && hist && hist_len > 0;
    h->history_len = use_hist || advance ? (hist ? hist_len : 0) : 0;
    h->history_window = window;
    h->history_count = h->history_len;
    h->step_idx = 0;
    h->advance = advance;
    h->temperature = sp ? sp->temperature : 0.f;
    h->penalty = sp ? sp->penalty : 1.f;
    h->r = r;
    h->out_token = -1;
    h->status = 0;
    if (h->history_len > 0) memcpy(h->history, hist, (size_t)h->history_len * sizeof(int));
    const size_t bytes = offsetof(StepState, history) + (size_t)h->history_len * sizeof(int);
    CU(cudaMemcpyAsync(e->st, h, bytes, cudaMemcpyHostToDevice, e->stream));
    return LPP_OK;
}

static lpp_status pull_result(lpp_engine* e, int* token) {
    TRACE("pull_result: waiting for the stream");
    CU(cudaMemcpyAsync(e->h_out, &e->st->out_token, 2 * sizeof(int), cudaMemcpyDeviceToHost, e->stream));
    CU(cudaStreamSynchronize(e->stream));
    if (e->h_out[1] != 0) return fail(LPP_ERR_DEVICE_STATUS, "device status 0x%x (1=barrier timeout, 2=bad token, 4=bad pos)", e->h_out[1]);
    if (token) *token = e->h_out[0];
    return LPP_OK;
}

// n tokens at positions start_pos .. are about to run: a recurrent state must stand at start_pos (or start anew at 0).  Until
// state_ran confirms that they have run, the state counts as unknown.
static lpp_status state_runs(lpp_engine* e, int start_pos) {
    if (!e->recurrent) return LPP_OK;
    if (start_pos != 0 && start_pos != e->state_len)
        return e->state_len < 0 ? fail(LPP_ERR_INVALID_ARG, "position %d: the recurrent state is not that of a sequence, start at position 0", start_pos)
                                : fail(LPP_ERR_INVALID_ARG, "position %d: the recurrent state stands at position %d", start_pos, e->state_len);
    e->state_len = -1;
    return LPP_OK;
}
static lpp_status state_ran(lpp_engine* e, int end_pos) {
    if (e->recurrent) e->state_len = end_pos;
    return LPP_OK;
}

#define NEED_READY(e)                                                              \
    do {                                                                           \
        if (!(e)) return fail(LPP_ERR_INVALID_ARG, "null engine");                 \
        if (!(e)->finalized) return fail(LPP_ERR_NOT_READY, "lpp_finalize not called"); \
        CU(cudaSetDevice((e)->c.device));                                          \
    } while (0)

extern "C" lpp_status lpp_step(lpp_engine* e, int token, int pos, const lpp_sample_params* sp, const int* h_history,
                               int history_len, float r, int* next_token) {
    NEED_READY(e);
    if (!sp || !next_token) return fail(LPP_ERR_INVALID_ARG, "null argument");
    TRY(push_state(e, token, pos, sp, h_history, history_len, r, 0, 0));
    TRY(state_runs(e, pos));
    TRY(run_step(e, true, pos));
    TRY(pull_result(e, next_token));
    return state_ran(e, pos + 1);
}

extern "C" lpp_status lpp_step_logits(lpp_engine* e, int token, int pos, float* h_logits) {
    NEED_READY(e);
    if (!h_logits) return fail(LPP_ERR_INVALID_ARG, "null argument");
    TRY(push_state(e, token, pos, nullptr, nullptr, 0, 0.f, 0, 0));
    TRY(state_runs(e, pos));
    TRY(run_step(e, false, pos));
    CU(cudaMemcpyAsync(h_logits, e->logits, (size_t)e->c.vocab_size * 4, cudaMemcpyDeviceToHost, e->stream));
    TRY(pull_result(e, nullptr));
    return state_ran(e, pos + 1);
}

extern "C" lpp_status lpp_decode(lpp_engine* e, int first_token, int start_pos, int n, const lpp_sample_params* sp,
                                 const int* h_history, int history_len, int history_window, const float* h_r,
                                 int* h_out_tokens, float* device_ms) {
    NEED_READY(e);
    if (!sp || !h_out_tokens || n <= 0) return fail(LPP_ERR_INVALID_ARG, "bad argument");
    if (n > e->run_cap) return fail(LPP_ERR_TOO_LARGE, "n %d > capacity %d", n, e->run_cap);
    if (start_pos + n > e->c.seq_len) return fail(LPP_ERR_INVALID_ARG, "start_pos + n exceeds seq_len %d", e->c.seq_len);
    if (history_window < 0 || history_window > kHistoryMax || history_len > std::max(history_window, 0))
        return fail(LPP_ERR_INVALID_ARG, "history_len %d / window %d invalid", history_len, history_window);
    if (sp->temperature != 0.0f && !h_r) return fail(LPP_ERR_INVALID_ARG, "temperature > 0 needs h_r");
    TRY(push_state(e, first_token, start_pos, sp, h_history, history_len, 0.f, 1, history_window));
    if (h_r) CU(cudaMemcpyAsync(e->r_values, h_r, (size_t)n * 4, cudaMemcpyHostToDevice, e->stream));
    TRY(state_runs(e, start_pos));
    CU(cudaEventRecord(e->ev0, e->stream));
    for (int i = 0; i < n; ++i) TRY(run_step(e, true, start_pos + i));
    CU(cudaEventRecord(e->ev1, e->stream));
    CU(cudaMemcpyAsync(h_out_tokens, e->out_tokens, (size_t)n * 4, cudaMemcpyDeviceToHost, e->stream));
    TRY(pull_result(e, nullptr));
    TRY(state_ran(e, start_pos + n));
    if (device_ms) CU(cudaEventElapsedTime(device_ms, e->ev0, e->ev1));
    return LPP_OK;
}

extern "C" lpp_status lpp_sample_logits(lpp_engine* e, const float* h_logits, const lpp_sample_params* sp,
                                        const int* h_history, int history_len, float r, int* token) {
    NEED_READY(e);
    if (!h_logits || !sp || !token) return fail(LPP_ERR_INVALID_ARG, "null argument");
    TRY(push_state(e, 0, 0, sp, h_history, history_len, r, 0, 0));
    CU(cudaMemcpyAsync(e->logits, h_logits, (size_t)e->c.vocab_size * 4, cudaMemcpyHostToDevice, e->stream));
    CU(launch_sampler(e, e->stream, false));
    return pull_result(e, token);
}

// ------------------------------------------------------------------ batched prompt path

typedef CUresult (*encode_tiled_fn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                    const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                    CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

static encode_tiled_fn tensor_map_encoder() {
    static encode_tiled_fn encode = nullptr;
    if (!encode) {
        cudaDriverEntryPointQueryResult qr;
        void* fn = nullptr;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &fn, cudaEnableDefault, &qr) == cudaSuccess && fn &&
            qr == cudaDriverEntryPointSuccess)
            encode = (encode_tiled_fn)fn;
    }
    return encode;
}

// Tensor maps over row-major FP16 matrices of THIS GPU's memory, cut into pieces of 64 inputs (128 bytes, stored with
// the 128-byte swizzle: the K-major operand layout of the MMA descriptors).  cols must be a multiple of 64; elements
// outside the matrix read as zero.
//
// Weights [rows][cols] seen as (64 inputs, rows, cols / 64): a box is 64 inputs x box_rows rows x 2 pieces, i.e. one
// copy delivers both 64-input sub-tiles of a stage, sub-tile after sub-tile.
static lpp_status make_weight_map(CUtensorMap* m, const void* base, size_t rows, size_t cols, int box_rows) {
    encode_tiled_fn encode = tensor_map_encoder();
    if (!encode) return fail(LPP_ERR_CUDA, "cuTensorMapEncodeTiled is not available from this driver");
    const cuuint64_t dims[3] = {64, (cuuint64_t)rows, (cuuint64_t)(cols / 64)};
    const cuuint64_t strides[2] = {(cuuint64_t)cols * 2, 128};
    const cuuint32_t box[3] = {64u, (cuuint32_t)box_rows, 2u};
    const cuuint32_t estr[3] = {1, 1, 1};
    const CUresult r = encode(m, CU_TENSOR_MAP_DATA_TYPE_FLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr,
                              CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                              CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) return fail(LPP_ERR_CUDA, "cuTensorMapEncodeTiled failed (%d) for a %zu x %zu matrix", (int)r, rows, cols);
    return LPP_OK;
}
// Activations: hi plane [tokens][cols] followed by the lo plane, seen as (64 inputs, tokens, 2 planes, cols / 64): a
// box is 64 inputs x box_tokens x 2 planes x 2 pieces, i.e. one copy delivers, per 64-input piece, the hi rows
// followed by the lo rows: one K-major operand tile of 2 x box_tokens rows (the MMA's N) per piece.
static lpp_status make_activation_map(CUtensorMap* m, const void* base, size_t tokens, size_t cols, int box_tokens) {
    encode_tiled_fn encode = tensor_map_encoder();
    if (!encode) return fail(LPP_ERR_CUDA, "cuTensorMapEncodeTiled is not available from this driver");
    const cuuint64_t dims[4] = {64, (cuuint64_t)tokens, 2, (cuuint64_t)(cols / 64)};
    const cuuint64_t strides[3] = {(cuuint64_t)cols * 2, (cuuint64_t)tokens * cols * 2, 128};
    const cuuint32_t box[4] = {64u, (cuuint32_t)box_tokens, 2u, 2u};
    const cuuint32_t estr[4] = {1, 1, 1, 1};
    const CUresult r = encode(m, CU_TENSOR_MAP_DATA_TYPE_FLOAT16, 4, const_cast<void*>(base), dims, strides, box, estr,
                              CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                              CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) return fail(LPP_ERR_CUDA, "cuTensorMapEncodeTiled failed (%d) for a %zu x %zu activation block", (int)r, tokens, cols);
    return LPP_OK;
}

// The tensor-core path takes 16-bit weights, an FP16 cache and a single GPU; everything else is fed token by token.
static bool prefill_batched(const lpp_engine* e) {
    if (e->c.flags & LPP_FLAG_NO_PREFILL_GEMM) return false;
    if (!e->layers.empty()) return e->c.weight_dtype == LPP_BF16 && e->c.kv_dtype == LPP_F16;
    return e->c.tp_size == 1 && e->c.weight_dtype == LPP_F16 && e->c.kv_dtype == LPP_F16 && e->hs <= 128 && e->gqa <= 8 &&
           e->c.dim % 64 == 0 && e->Dq % 64 == 0 && e->Fl % 64 == 0;
}

template <typename T>
static lpp_status allow_gemm_smem() {
    CU(cudaFuncSetAttribute(prefill_gemm_umma_kernel<T, kPfResid>, cudaFuncAttributeMaxDynamicSharedMemorySize, kPfSmemBytes));
    CU(cudaFuncSetAttribute(prefill_gemm_umma_kernel<T, kPfSwiglu>, cudaFuncAttributeMaxDynamicSharedMemorySize, kPfSmemBytes));
    CU(cudaFuncSetAttribute(prefill_gemm_umma_kernel<T, kPfStore>, cudaFuncAttributeMaxDynamicSharedMemorySize, kPfSmemBytes));
    return LPP_OK;
}

static lpp_status prefill_setup(lpp_engine* e) {
    if (e->pf_ready) return LPP_OK;
    const lpp_config& c = e->c;
    const size_t D = e->Dp, L = c.n_layers, T = kPrefillTokens;
    const bool layered = !e->layers.empty();
    size_t part_rows = D, att_n = e->Dq, hb_n = e->Fl, qn_n = 0, olat_n = 0, lq_n = 0, lpart_n = 0, gate_n = 0, scan_n = 0, tail_n = 0, low_n = 0;
    const size_t qkv_rows = layered ? 0 : e->Dq + 2 * (size_t)e->KVd;
    part_rows = std::max(part_rows, qkv_rows);
    for (const ModelLayer& y : e->layers) {
        const size_t H = y.d.heads;
        part_rows = std::max(part_rows, (size_t)y.in_rows);
        att_n = std::max(att_n, (size_t)y.o_pitch);
        hb_n = std::max(hb_n, (size_t)y.ff_pitch);
        if (y.d.mixer == LPP_MIXER_MAMBA) {
            part_rows = std::max(part_rows, (size_t)y.low_rows * kLowMaxSplits / kPfMaxSplits);
            low_n = std::max(low_n, (size_t)mamba_low_pitch(y.dt_pitch, y.state_pitch));
            scan_n = std::max(scan_n, (size_t)y.inner_pitch);
            tail_n = std::max(tail_n, (size_t)(y.d.conv - 1) * y.inner_rows);
            continue;
        }
        if (y.d.mixer == LPP_MIXER_LATENT) {
            qn_n = std::max(qn_n, H * y.dim_pitch);
            olat_n = std::max(olat_n, H * y.val_pitch);
        }
        lq_n = std::max(lq_n, H * y.row_width);
        for (size_t t = 1; t <= T; ++t) {
            const LatentPlan p = latent_plan(e, y, (int)t);
            if (!p.cluster) lpart_n = std::max(lpart_n, t * H * p.splits * (y.rank_pitch + kLatentPartTail));
        }
        gate_n = std::max(gate_n, y.d.mixer == LPP_MIXER_LATENT ? H : H * y.d.dim);
    }
    TRY(zeroed(e, &e->pf_x, T * D * 4));
    TRY(zeroed(e, &e->pf_xn, 2 * T * D * 2));      // hi plane, lo plane
    TRY(zeroed(e, &e->pf_att, 2 * T * att_n * 2));  // hi plane, lo plane
    TRY(zeroed(e, &e->pf_hb, 2 * T * hb_n * 2));    // hi plane, lo plane
    TRY(zeroed(e, &e->pf_part, (size_t)kPfMaxSplits * T * part_rows * 4));
    TRY(zeroed(e, &e->pf_tokens, T * sizeof(int)));
    TRY(zeroed(e, &e->pf_rows, T * sizeof(int)));
    if (layered) {
        TRY(zeroed(e, &e->pf_qn, 2 * T * qn_n * 2));
        TRY(zeroed(e, &e->pf_olat, 2 * T * olat_n * 2));
        TRY(zeroed(e, &e->pf_lq, T * lq_n * 2));
        TRY(zeroed(e, &e->pf_lpart, lpart_n * 4));
        TRY(zeroed(e, &e->pf_gate, T * gate_n * 4));
        TRY(zeroed(e, &e->pf_sx, T * scan_n * 4));
        TRY(zeroed(e, &e->pf_sz, T * scan_n * 4));
        TRY(zeroed(e, &e->pf_sxp, 2 * T * scan_n * 2));
        TRY(zeroed(e, &e->pf_tail, tail_n * 4));
        TRY(zeroed(e, &e->pf_low, T * low_n * 4));
        for (ModelLayer& y : e->layers) {
            const size_t H = y.d.heads, D2 = align_up(c.dim, 2);
            TRY(make_weight_map(&y.m_in, y.w_in, y.in_rows, D, kUmmaM));
            if (y.d.mixer == LPP_MIXER_LATENT) {
                TRY(make_weight_map(&y.m_uk, y.w_uk, H * y.rank_pitch, y.dim_pitch, kUmmaM));
                TRY(make_weight_map(&y.m_uv, y.w_uv, H * y.vdim_rows, y.val_pitch, kUmmaM));
                TRY(make_activation_map(&y.x_qn, e->pf_qn, T, H * y.dim_pitch, kPrefillTokens));
                TRY(make_activation_map(&y.x_olat, e->pf_olat, T, H * y.val_pitch, kPrefillTokens));
            } else if (y.d.mixer == LPP_MIXER_MAMBA) {
                TRY(make_weight_map(&y.m_low, y.w_low, y.low_rows, y.inner_pitch, kUmmaM));
                TRY(make_activation_map(&y.x_low, e->pf_sxp, T, y.inner_pitch, kPrefillTokens));
            }
            TRY(make_weight_map(&y.m_wo, y.wo, D2, y.o_pitch, kUmmaM));
            TRY(make_activation_map(&y.x_att, e->pf_att, T, y.o_pitch, kPrefillTokens));
            if (y.d.ff > 0) {
                TRY(make_weight_map(&y.m_w13, y.w13, 2 * (size_t)y.d.ff, D, kUmmaM));
                TRY(make_weight_map(&y.m_w2, y.w2, D2, y.ff_pitch, kUmmaM));
                TRY(make_activation_map(&y.x_hb, e->pf_hb, T, y.ff_pitch, kPrefillTokens));
            }
        }
        TRY(allow_gemm_smem<__nv_bfloat16>());
        CU(cudaFuncSetAttribute(prefill_gemm_umma_kernel<__nv_bfloat16, kPfLatentQuery>, cudaFuncAttributeMaxDynamicSharedMemorySize, kPfSmemBytes));
        CU(cudaFuncSetAttribute(prefill_gemm_umma_kernel<__nv_bfloat16, kPfLatentValue>, cudaFuncAttributeMaxDynamicSharedMemorySize, kPfSmemBytes));
    } else {
        TRY(zeroed(e, &e->pf_q, T * e->Dq * 4));
        TRY(make_weight_map(&e->pf_map_wqkv, e->wqkv, L * qkv_rows, D, kUmmaM));
        TRY(make_weight_map(&e->pf_map_wo, e->wo, L * D, e->Dq, kUmmaM));
        TRY(make_weight_map(&e->pf_map_w13, e->w13, L * 2 * e->Fl, D, kUmmaM));
        TRY(make_weight_map(&e->pf_map_w2, e->w2, L * D, e->Fl, kUmmaM));
        TRY(make_activation_map(&e->pf_map_att, e->pf_att, T, e->Dq, kPrefillTokens));
        TRY(make_activation_map(&e->pf_map_hb, e->pf_hb, T, e->Fl, kPrefillTokens));
        TRY(allow_gemm_smem<__half>());
        CU(cudaFuncSetAttribute(prefill_gemm_umma_kernel<__half, kPfQkv>, cudaFuncAttributeMaxDynamicSharedMemorySize, kPfSmemBytes));
        CU(cudaFuncSetAttribute(prefill_attention_mma_kernel<64>, cudaFuncAttributeMaxDynamicSharedMemorySize, pf_attn_smem<64>()));
        CU(cudaFuncSetAttribute(prefill_attention_mma_kernel<128>, cudaFuncAttributeMaxDynamicSharedMemorySize, pf_attn_smem<128>()));
    }
    TRY(make_activation_map(&e->pf_map_xn, e->pf_xn, T, D, kPrefillTokens));
    TRY(make_weight_map(&e->pf_map_cls, e->wcls, e->Vp, D, kUmmaM));
    e->pf_ready = true;
    return LPP_OK;
}

// Ranges of K a GEMM is cut into so that its row tiles (128 weight rows: the weight maps' box) fill the GPU.
static int prefill_splits(const lpp_engine* e, int n_rows, int K, int max_splits = kPfMaxSplits) {
    const int tiles = (n_rows + kUmmaM - 1) / kUmmaM, n_kc = (K + kPfKc - 1) / kPfKc;
    return tiles < e->num_sms ? std::max(1, std::min({max_splits, n_kc, (e->num_sms + tiles - 1) / tiles})) : 1;
}

// A GEMM whose row tiles do not fill the GPU is also cut along K (a.splits); its partial sums go to pf_part and are added
// up by the next prefill_norm_kernel (residual projections) or by a finishing kernel (input projections).
template <typename T, int EPI>
static cudaError_t launch_prefill_gemm_t(lpp_engine* e, const CUtensorMap& wm, const CUtensorMap& xm, const PrefillGemmArgs& a) {
    const int tiles = (a.n_rows + kUmmaM - 1) / kUmmaM * std::max(1, a.groups);
    return launch_kernel(prefill_gemm_umma_kernel<T, EPI>, dim3(std::min(tiles * a.splits, e->num_sms)), dim3(kUmmaThreads),
                         (size_t)kPfSmemBytes, e->stream, true, wm, xm, a);
}
template <int EPI>
static cudaError_t launch_prefill_gemm(lpp_engine* e, const CUtensorMap& wm, const CUtensorMap& xm, const PrefillGemmArgs& a) {
    return e->c.weight_dtype == LPP_BF16 ? launch_prefill_gemm_t<__nv_bfloat16, EPI>(e, wm, xm, a)
                                         : launch_prefill_gemm_t<__half, EPI>(e, wm, xm, a);
}
static PrefillGemmArgs prefill_gemm_args(const lpp_engine* e, int n_rows, int K, int n_tokens, int start_pos) {
    PrefillGemmArgs a = {};
    a.n_rows = n_rows;
    a.K = K;
    a.n_tokens = n_tokens;
    a.start_pos = start_pos;
    a.splits = 1;
    a.part = e->pf_part;
    a.st = e->st;
    return a;
}

// x_rows -> normalised operands; `parts` > 1: the previous residual GEMM's partial sums are added to x first, and so is `add`
// (nullptr = nothing).
static lpp_status prefill_norm(lpp_engine* e, int n, const float* w, const float* b, bool embed, const float* add, int parts, const int* rows, bool pdl) {
    PrefillNormArgs a = {};
    a.x = e->pf_x;
    a.tokens = e->pf_tokens;
    a.emb = embed ? e->emb : nullptr;
    a.emb_scale = e->emb_scale;
    a.add = add;
    a.vocab = e->c.vocab_size;
    a.rows = rows;
    a.norm_w = w;
    a.norm_b = b;
    a.norm_eps = e->norm_eps;
    a.norm_n = e->c.dim;
    a.out = e->pf_xn;
    a.D = e->Dp;
    a.part = e->pf_part;
    a.splits = embed ? 1 : parts;
    a.st = e->st;
    if (e->c.weight_dtype == LPP_BF16)
        CU(launch_kernel(prefill_norm_kernel<__nv_bfloat16>, dim3(n), dim3(kPfNormThreads), 0, e->stream, pdl, a));
    else
        CU(launch_kernel(prefill_norm_kernel<__half>, dim3(n), dim3(kPfNormThreads), 0, e->stream, pdl, a));
    return LPP_OK;
}

// x += W . in  for the block: output and down projection.  Returns the number of partial sums the next norm adds.
static lpp_status prefill_resid(lpp_engine* e, const CUtensorMap& wm, int row0, const CUtensorMap& xm, int K, int n, int start_pos, int* parts) {
    // all Dp columns: beyond dim the products are zero (rows outside the map), and so are the partial sums that the norm adds
    PrefillGemmArgs g = prefill_gemm_args(e, e->Dp, K, n, start_pos);
    g.row0 = row0;
    g.x = e->pf_x;
    g.x_pitch = e->Dp;
    g.splits = *parts = prefill_splits(e, g.n_rows, K);
    CU(launch_prefill_gemm<kPfResid>(e, wm, xm, g));
    return LPP_OK;
}

// Grouped-query attention of a prompt block: K/V rows to the cache and, unless only those are wanted, the attended values
// to pf_att.
static lpp_status prefill_gqa_mixer(lpp_engine* e, int l, int n, int start_pos, bool cache_only) {
    const lpp_config& c = e->c;
    const int D = c.dim, qkv_rows = e->Dq + 2 * e->KVd;
    const size_t lofs = (size_t)l * e->KVHl * c.seq_len * e->hs;
    PrefillGemmArgs g = prefill_gemm_args(e, qkv_rows, D, n, start_pos);
    g.row0 = l * qkv_rows;
    g.epi = kPfQkv;
    g.q = e->pf_q;
    g.q_rows = e->Dq;
    g.kv_rows = e->KVd;
    g.head_size = e->hs;
    g.seq_len = c.seq_len;
    g.rope = e->rope;
    g.k_cache = (__half*)e->kcache + lofs;
    g.v_cache = (__half*)e->vcache + lofs;
    g.splits = prefill_splits(e, qkv_rows, D);
    const cudaError_t ge = launch_prefill_gemm_t<__half, kPfQkv>(e, e->pf_map_wqkv, e->pf_map_xn, g);
    CU(ge);
    if (g.splits > 1)
        CU(launch_kernel(prefill_qkv_finish_kernel, dim3(n, (qkv_rows / 2 + 255) / 256), dim3(256), 0, e->stream, true, g));
    if (cache_only) return LPP_OK;
    const dim3 agrid((n + kPfAttnRows - 1) / kPfAttnRows, e->KVHl);
    __half* att = (__half*)e->pf_att;
    const bool pf_mma = !aid_env("LPP_ATTN_CUDA_CORES");
    if (pf_mma && e->hs == 64 && e->gqa <= 8)
        CU(launch_kernel(prefill_attention_mma_kernel<64>, agrid, dim3(32 * e->gqa), pf_attn_smem<64>(), e->stream, true,
                         (const float*)e->pf_q, (const __half*)g.k_cache, (const __half*)g.v_cache, att, n, start_pos,
                         c.seq_len, e->gqa, e->Dq));
    else if (pf_mma && e->hs == 128 && e->gqa <= 8)
        CU(launch_kernel(prefill_attention_mma_kernel<128>, agrid, dim3(32 * e->gqa), pf_attn_smem<128>(), e->stream, true,
                         (const float*)e->pf_q, (const __half*)g.k_cache, (const __half*)g.v_cache, att, n, start_pos,
                         c.seq_len, e->gqa, e->Dq));
    else
        CU(launch_kernel(prefill_attention_kernel, dim3(n, e->KVHl), dim3(32 * e->gqa),
                         (size_t)e->gqa * e->hs * sizeof(float), e->stream, true, (const float*)e->pf_q,
                         (const __half*)g.k_cache, (const __half*)g.v_cache, att, n, start_pos, c.seq_len, e->hs,
                         e->gqa, e->Dq));
    return LPP_OK;
}

// W . in of a block as partial sums over ranges of K, [range][token][row] in pf_part; *splits = the number of ranges.
static lpp_status prefill_partial_sums(lpp_engine* e, const CUtensorMap& wm, const CUtensorMap& xm, int n_rows, int K, int n, int start_pos, int* splits,
                                       int max_splits = kPfMaxSplits) {
    PrefillGemmArgs g = prefill_gemm_args(e, n_rows, K, n, start_pos);
    g.out = e->pf_part;
    g.out_pitch = n_rows;
    g.splits = *splits = prefill_splits(e, n_rows, K, max_splits);
    CU((launch_prefill_gemm_t<__nv_bfloat16, kPfStore>(e, wm, xm, g)));
    return LPP_OK;
}

// Attention over shared rows of a prompt block: queries pf_lq, finished rows to `planes` as hi + lo operands.
static lpp_status prefill_row_attention(lpp_engine* e, const ModelLayer& y, const LayerRun& r, int n, int start_pos, void* planes) {
    const LatentPlan p = latent_plan(e, y, n);
    LatentAttnArgs a = latent_attn_args(e, y, r, p);
    a.q = e->pf_lq;
    a.part = e->pf_lpart;
    a.start_pos = start_pos;
    a.n_tokens = n;
    a.planes = (__nv_bfloat16*)planes;
    a.out = nullptr;
    if (a.gate) a.gate = e->pf_gate;
    CU(launch_latent_attn(e, p, a, y.d.mixer == LPP_MIXER_SHARED_KV, true, e->stream));
    if (!p.cluster)
        CU(launch_kernel(prefill_latent_combine_kernel, dim3(n * a.all_heads), dim3(128), 0, e->stream, true, a, p.tile_rows));
    return LPP_OK;
}

// Latent attention of a prompt block: input GEMM (cut along K) and its finishing kernel, per-head query GEMM, attention in
// key splits, their combination, per-head value GEMM with the gates.
static lpp_status prefill_latent_mixer(lpp_engine* e, int l, int n, int start_pos, bool cache_only) {
    typedef __nv_bfloat16 T;
    const LayerRun& r = e->runs[l];
    const ModelLayer& y = e->layers[r.layer];
    const int H = y.d.heads;
    PrefillLatentFinishArgs f = {};
    TRY(prefill_partial_sums(e, y.m_in, e->pf_map_xn, y.in_rows, e->Dp, n, start_pos, &f.splits));
    f.part = e->pf_part;
    f.n_rows = y.in_rows;
    f.start_pos = start_pos;
    f.seq_len = e->c.seq_len;
    f.qn = e->pf_qn;
    f.gate = e->pf_gate;
    f.st = e->st;
    f.lat = latent_args(e, y, r);
    f.lat.query = e->pf_lq;
    const int q_sections = cache_only ? 0 : (y.q_plain_rows + y.q_rot_rows + 2 * kLatFinishThreads - 1) / (2 * kLatFinishThreads);
    CU(launch_kernel(prefill_latent_finish_kernel<T>, dim3(n, 1 + q_sections), dim3(kLatFinishThreads), (size_t)y.latent_rows * 4, e->stream,
                     true, f));
    if (cache_only) return LPP_OK;
    PrefillGemmArgs q = prefill_gemm_args(e, y.rank_pitch, y.dim_pitch, n, start_pos);
    q.groups = H;
    q.group_stride = y.rank_pitch;
    q.group_pieces = y.dim_pitch / 64;
    q.lat_query = e->pf_lq;
    q.lat_pitch = y.row_width;
    CU((launch_prefill_gemm_t<T, kPfLatentQuery>(e, y.m_uk, y.x_qn, q)));
    TRY(prefill_row_attention(e, y, r, n, start_pos, e->pf_olat));
    PrefillGemmArgs v = prefill_gemm_args(e, y.vdim_rows, y.val_pitch, n, start_pos);
    v.groups = H;
    v.group_stride = y.vdim_rows;
    v.group_pieces = y.val_pitch / 64;
    v.hb = e->pf_att;
    v.hb_pitch = y.o_pitch;
    v.gate = e->pf_gate;
    v.n_valid = y.d.vdim;
    CU((launch_prefill_gemm_t<T, kPfLatentValue>(e, y.m_uv, y.x_olat, v)));
    return LPP_OK;
}

// Attention whose values are its keys, of a prompt block: input GEMM (cut along K) and its finishing kernel, attention.
static lpp_status prefill_shared_kv_mixer(lpp_engine* e, int l, int n, int start_pos, bool cache_only) {
    const LayerRun& r = e->runs[l];
    const ModelLayer& y = e->layers[r.layer];
    PrefillSharedKvArgs f = {};
    TRY(prefill_partial_sums(e, y.m_in, e->pf_map_xn, y.in_rows, e->Dp, n, start_pos, &f.splits));
    f.part = e->pf_part;
    f.n_rows = y.in_rows;
    f.start_pos = start_pos;
    f.seq_len = e->c.seq_len;
    f.keys_only = cache_only;
    f.st = e->st;
    f.kv = shared_kv_args(e, y, r);
    f.kv.query = e->pf_lq;
    f.kv.gate = e->pf_gate;
    CU(launch_kernel(prefill_shared_kv_finish_kernel, dim3(n, (y.in_rows / 2 + 255) / 256), dim3(256), 0, e->stream, true, f));
    return cache_only ? LPP_OK : prefill_row_attention(e, y, r, n, start_pos, e->pf_att);
}

// Selective scan of a prompt block: input GEMM (cut along K), convolution, GEMM of dt | B | C (cut along K), recurrence.
static lpp_status prefill_mamba_mixer(lpp_engine* e, int l, int n, int start_pos) {
    const LayerRun& r = e->runs[l];
    const ModelLayer& y = e->layers[r.layer];
    MambaConvArgs v = {};
    TRY(prefill_partial_sums(e, y.m_in, e->pf_map_xn, y.in_rows, e->Dp, n, start_pos, &v.splits));
    v.part = e->pf_part;
    v.n_tokens = n;
    v.start_pos = start_pos;
    v.seq_len = e->c.seq_len;
    v.inner = y.d.inner;
    v.inner_rows = y.inner_rows;
    v.taps = y.d.conv;
    v.conv_w = y.conv_w;
    v.conv_b = y.conv_b;
    v.ring = r.ring;
    v.tail = e->pf_tail;
    v.x = e->pf_sx;
    v.z = e->pf_sz;
    v.x_pitch = y.inner_pitch;
    v.planes = (__nv_bfloat16*)e->pf_sxp;
    v.st = e->st;
    CU(launch_mamba_conv(v, e->stream));
    MambaScanArgs a = mamba_scan_args(e, y, r);
    int splits;
    TRY(prefill_partial_sums(e, y.m_low, y.x_low, y.low_rows, y.inner_pitch, n, start_pos, &splits, kLowMaxSplits));
    CU(launch_kernel(mamba_low_kernel, dim3(n, (y.dt_pitch + 2 * y.state_pitch + kLowColumns - 1) / kLowColumns), dim3(kLowThreads), 0, e->stream, true,
                     a, (const float*)e->pf_part, splits, e->pf_low));
    a.low = e->pf_low;
    a.n_tokens = n;
    a.start_pos = start_pos;
    a.x = e->pf_sx;
    a.z = e->pf_sz;
    a.x_pitch = y.inner_pitch;
    a.tail = e->pf_tail;
    a.planes = (__nv_bfloat16*)e->pf_att;
    a.plane_row = y.o_pitch;
    CU(launch_mamba_scan(e, a, e->stream));
    return LPP_OK;
}

// One block of n <= kPrefillTokens prompt tokens at positions start_pos ...  Without wanted logits the last layer stops
// after its cache rows are written (nothing downstream of them is needed); otherwise the n_want rows `want` of the block go
// through the final norm and the classifier and their logits are copied to h_logits.
static lpp_status prefill_block(lpp_engine* e, const int* h_tokens, int n, int start_pos, const int* want, int n_want, float* h_logits) {
    const lpp_config& c = e->c;
    const int L = n_runs(e);
    const bool layered = !e->layers.empty();
    CU(cudaMemcpyAsync(e->pf_tokens, h_tokens, (size_t)n * sizeof(int), cudaMemcpyHostToDevice, e->stream));
    if (n_want > 0) CU(cudaMemcpyAsync(e->pf_rows, want, (size_t)n_want * sizeof(int), cudaMemcpyHostToDevice, e->stream));
    int parts = 1;
    const float* add = first_add(e);  // what the next norm adds to the residual stream first
    for (int l = 0; l < L; ++l) {
        const bool cache_only = l == L - 1 && n_want == 0;
        const LayerView v = layer_view(e, l);
        const ModelLayer* y = layered ? &e->layers[e->runs[l].layer] : nullptr;
        // layer 0 takes the embedding rows; later layers first add the previous residual GEMM's partial sums
        TRY(prefill_norm(e, n, layered ? y->n1w : e->rms_att + (size_t)l * c.dim, layered ? y->n1b : nullptr, l == 0, add, parts, nullptr, l > 0));
        if (!layered)
            TRY(prefill_gqa_mixer(e, l, n, start_pos, cache_only));
        else if (y->d.mixer == LPP_MIXER_LATENT)
            TRY(prefill_latent_mixer(e, l, n, start_pos, cache_only));
        else if (y->d.mixer == LPP_MIXER_SHARED_KV)
            TRY(prefill_shared_kv_mixer(e, l, n, start_pos, cache_only));
        else
            TRY(prefill_mamba_mixer(e, l, n, start_pos));
        if (cache_only) return LPP_OK;
        TRY(prefill_resid(e, layered ? y->m_wo : e->pf_map_wo, layered ? 0 : l * c.dim, layered ? y->x_att : e->pf_map_att, v.o_k, n, start_pos,
                          &parts));
        add = v.o_add;
        if (v.ff == 0) continue;  // a layer without a feed-forward
        TRY(prefill_norm(e, n, v.norm2_w, v.norm2_b, false, add, parts, nullptr, true));
        PrefillGemmArgs u = prefill_gemm_args(e, 2 * v.ff, e->Dp, n, start_pos);
        u.row0 = layered ? 0 : l * 2 * v.ff;
        u.hb = e->pf_hb;
        u.hb_pitch = v.ff_k;
        u.act = v.act;
        CU(launch_prefill_gemm<kPfSwiglu>(e, layered ? y->m_w13 : e->pf_map_w13, e->pf_map_xn, u));
        TRY(prefill_resid(e, layered ? y->m_w2 : e->pf_map_w2, layered ? 0 : l * c.dim, layered ? y->x_hb : e->pf_map_hb, v.ff_k, n, start_pos,
                          &parts));
        add = v.down_add;
    }
    if (!e->pf_logits) CU(cudaMalloc(&e->pf_logits, (size_t)kPrefillTokens * e->Vp * 4));
    TRY(prefill_norm(e, n_want, e->rms_final, e->final_b, false, add, parts, e->pf_rows, true));
    PrefillGemmArgs g = prefill_gemm_args(e, e->Vp, e->Dp, n_want, start_pos);
    g.out = e->pf_logits;
    g.out_pitch = e->Vp;
    CU(launch_prefill_gemm<kPfStore>(e, e->pf_map_cls, e->pf_map_xn, g));
    CU(cudaMemcpy2DAsync(h_logits, (size_t)c.vocab_size * 4, e->pf_logits, (size_t)e->Vp * 4, (size_t)c.vocab_size * 4, n_want,
                         cudaMemcpyDeviceToHost, e->stream));
    return LPP_OK;
}

extern "C" lpp_status lpp_extend(lpp_engine* e, const int* h_tokens, int n, int start_pos, const int* want, int n_want, float* h_logits,
                                 float* device_ms) {
    NEED_READY(e);
    if (!h_tokens || n <= 0 || n_want < 0 || (n_want > 0 && (!want || !h_logits))) return fail(LPP_ERR_INVALID_ARG, "bad argument");
    if (start_pos < 0 || start_pos > e->c.seq_len - n) return fail(LPP_ERR_INVALID_ARG, "positions %d..%d outside [0, %d)", start_pos, start_pos + n - 1, e->c.seq_len);
    for (int i = 0; i < n; ++i)
        if (h_tokens[i] < 0 || h_tokens[i] >= e->c.vocab_size) return fail(LPP_ERR_INVALID_ARG, "token %d outside [0, %d)", h_tokens[i], e->c.vocab_size);
    for (int i = 0; i < n_want; ++i)
        if (want[i] < (i ? want[i - 1] + 1 : 0) || want[i] >= n) return fail(LPP_ERR_INVALID_ARG, "wanted tokens must ascend within the portion");
    const size_t V = e->c.vocab_size;
    int w = 0;  // wanted tokens served so far
    TRY(push_state(e, h_tokens[0], start_pos, nullptr, nullptr, 0, 0.f, 0, 0));  // clears the device status
    TRY(state_runs(e, start_pos));
    if (prefill_batched(e) && n > 1) {
        TRY(prefill_setup(e));
        CU(cudaEventRecord(e->ev0, e->stream));
        for (int i = 0; i < n; i += kPrefillTokens) {
            const int m = std::min(kPrefillTokens, n - i);
            int rows[kPrefillTokens], k = 0;
            while (w + k < n_want && want[w + k] < i + m) rows[k] = want[w + k] - i, ++k;
            TRY(prefill_block(e, h_tokens + i, m, start_pos + i, rows, k, h_logits + (size_t)w * V));
            w += k;
        }
        CU(cudaEventRecord(e->ev1, e->stream));
    } else {
        // token by token through the step graph without its sampler, like the reference's prompt loop
        CU(cudaEventRecord(e->ev0, e->stream));
        for (int i = 0; i < n; ++i) {
            if (i > 0) TRY(push_state(e, h_tokens[i], start_pos + i, nullptr, nullptr, 0, 0.f, 0, 0));
            TRY(run_step(e, false, start_pos + i));
            if (w < n_want && want[w] == i)
                CU(cudaMemcpyAsync(h_logits + (size_t)w++ * V, e->logits, V * 4, cudaMemcpyDeviceToHost, e->stream));
            // the pinned staging block of push_state is rewritten by the next token (the copy must have run), and the
            // next token's push would clear a status this one has set
            if (i + 1 < n) TRY(pull_result(e, nullptr));
        }
        CU(cudaEventRecord(e->ev1, e->stream));
    }
    TRY(pull_result(e, nullptr));
    TRY(state_ran(e, start_pos + n));
    if (device_ms) CU(cudaEventElapsedTime(device_ms, e->ev0, e->ev1));
    return LPP_OK;
}

extern "C" lpp_status lpp_prefill(lpp_engine* e, const int* h_tokens, int n, int start_pos, float* device_ms) {
    return lpp_extend(e, h_tokens, n, start_pos, nullptr, 0, nullptr, device_ms);
}

// ------------------------------------------------------------------ KV cache access

extern "C" int64_t lpp_kv_index(const lpp_engine* e, int layer, int kv_head, int pos, int off) {
    if (!e || !e->layers.empty()) return -1;
    const int64_t kvd = (int64_t)e->KVHl * e->hs, S = e->c.seq_len;
    return (int64_t)layer * (kvd * S) + (int64_t)kv_head * (S * e->hs) + (int64_t)pos * e->hs + off;
}

extern "C" lpp_status lpp_kv_prefill(lpp_engine* e, int layer, const void* k, const void* v, int n_pos, int src_dtype,
                                     int memkind) {
    if (!e || !k || !v) return fail(LPP_ERR_INVALID_ARG, "null argument");
    const lpp_config& c = e->c;
    if (!e->layers.empty()) return fail(LPP_ERR_INVALID_ARG, "this model keeps no separate keys and values");
    if (layer < 0 || layer >= c.n_layers || n_pos < 0 || n_pos > c.seq_len) return fail(LPP_ERR_INVALID_ARG, "layer/n_pos out of range");
    if (src_dtype != LPP_F16 && src_dtype != LPP_F32) return fail(LPP_ERR_INVALID_ARG, "bad src_dtype");
    CU(cudaSetDevice(c.device));
    const int hs = e->hs;
    for (int h = 0; h < e->KVHl; ++h) {
        const size_t gh = (size_t)c.tp_rank * e->KVHl + h;  // global kv head
        const size_t dst = (size_t)lpp_kv_index(e, layer, h, 0, 0) * e->kvesz;
        // source rows [gh][0..n_pos) are contiguous: one block of n_pos rows x hs columns
        TRY(put_block(e, (char*)e->kcache + dst, hs, c.kv_dtype, k, hs, gh * n_pos, 0, n_pos, hs, src_dtype, memkind));
        TRY(put_block(e, (char*)e->vcache + dst, hs, c.kv_dtype, v, hs, gh * n_pos, 0, n_pos, hs, src_dtype, memkind));
    }
    if (e->stage && e->finalized) {
        cudaFree(e->stage);
        e->stage = nullptr;
        e->stage_bytes = 0;
    }
    return LPP_OK;
}

extern "C" lpp_status lpp_kv_read(lpp_engine* e, int layer, int kv_head, int pos, float* h_k, float* h_v) {
    if (!e || !h_k || !h_v) return fail(LPP_ERR_INVALID_ARG, "null argument");
    const lpp_config& c = e->c;
    if (!e->layers.empty()) return fail(LPP_ERR_INVALID_ARG, "this model keeps no separate keys and values");
    if (layer < 0 || layer >= c.n_layers || kv_head < 0 || kv_head >= e->KVHl || pos < 0 || pos >= c.seq_len)
        return fail(LPP_ERR_INVALID_ARG, "index out of range");
    CU(cudaSetDevice(c.device));
    const size_t off = (size_t)lpp_kv_index(e, layer, kv_head, pos, 0) * e->kvesz;
    const int hs = e->hs;
    CU(cudaStreamSynchronize(e->stream));
    if (c.kv_dtype == LPP_F32) {
        CU(cudaMemcpy(h_k, (char*)e->kcache + off, hs * 4, cudaMemcpyDeviceToHost));
        CU(cudaMemcpy(h_v, (char*)e->vcache + off, hs * 4, cudaMemcpyDeviceToHost));
    } else {
        std::vector<__half> tk(hs), tv(hs);
        CU(cudaMemcpy(tk.data(), (char*)e->kcache + off, hs * 2, cudaMemcpyDeviceToHost));
        CU(cudaMemcpy(tv.data(), (char*)e->vcache + off, hs * 2, cudaMemcpyDeviceToHost));
        for (int i = 0; i < hs; ++i) {
            h_k[i] = __half2float(tk[i]);
            h_v[i] = __half2float(tv[i]);
        }
    }
    return LPP_OK;
}

extern "C" lpp_status lpp_latent_read(lpp_engine* e, int layer, int pos, float* h_row) {
    if (!e || !h_row) return fail(LPP_ERR_INVALID_ARG, "null argument");
    if (layer < 0 || layer >= (int)e->runs.size() || pos < 0 || pos >= e->c.seq_len) return fail(LPP_ERR_INVALID_ARG, "index out of range");
    const LayerRun& r = e->runs[layer];
    const ModelLayer& y = e->layers[r.layer];
    if (y.d.mixer != LPP_MIXER_LATENT) return fail(LPP_ERR_INVALID_ARG, "layer run %d keeps no latents", layer);
    CU(cudaSetDevice(e->c.device));
    CU(cudaStreamSynchronize(e->stream));
    std::vector<unsigned char> raw((size_t)y.row_width * e->kvesz);
    CU(cudaMemcpy(raw.data(), (const char*)r.cache + (size_t)pos * raw.size(), raw.size(), cudaMemcpyDeviceToHost));
    auto at = [&](int i) { return e->kvesz == 4 ? ((const float*)raw.data())[i] : __half2float(((const __half*)raw.data())[i]); };
    for (int i = 0; i < y.d.kv_rank; ++i) h_row[i] = at(i);
    for (int i = 0; i < y.d.rot_dim; ++i) h_row[y.d.kv_rank + i] = at(y.rank_pitch + i);
    return LPP_OK;
}

// ------------------------------------------------------------------ introspection

// ---- tensor-parallel peer mapping ---------------------------------------------------------------

static_assert(sizeof(cudaIpcMemHandle_t) == LPP_TP_HANDLE_BYTES, "IPC handle size");

extern "C" lpp_status lpp_tp_export(lpp_engine* e, void* handle, size_t handle_bytes) {
    if (!e || !handle) return fail(LPP_ERR_INVALID_ARG, "null argument");
    if (handle_bytes < sizeof(cudaIpcMemHandle_t)) return fail(LPP_ERR_INVALID_ARG, "handle buffer needs %zu bytes", sizeof(cudaIpcMemHandle_t));
    if (!e->tp_buf || e->c.tp_size < 2) return fail(LPP_ERR_INVALID_ARG, "engine has no tensor-parallel exchange buffer (tp_size 1 or > %d)", kMaxTp);
    CU(cudaSetDevice(e->c.device));
    cudaIpcMemHandle_t h;
    CU(cudaIpcGetMemHandle(&h, e->tp_buf));
    memcpy(handle, &h, sizeof h);
    return LPP_OK;
}

extern "C" lpp_status lpp_tp_connect(lpp_engine* e, const void* handles, size_t handle_bytes) {
    if (!e || !handles) return fail(LPP_ERR_INVALID_ARG, "null argument");
    if (handle_bytes < sizeof(cudaIpcMemHandle_t)) return fail(LPP_ERR_INVALID_ARG, "handles are %zu bytes each", sizeof(cudaIpcMemHandle_t));
    if (!e->tp_buf || e->c.tp_size < 2) return fail(LPP_ERR_INVALID_ARG, "engine has no tensor-parallel exchange buffer");
    if (e->finalized) return fail(LPP_ERR_INVALID_ARG, "lpp_tp_connect must precede lpp_finalize");
    CU(cudaSetDevice(e->c.device));
    for (int p = 0; p < e->c.tp_size; ++p) {
        if (p == e->c.tp_rank || e->peer_base[p]) continue;
        cudaIpcMemHandle_t h;
        memcpy(&h, (const char*)handles + (size_t)p * handle_bytes, sizeof h);
        void* ptr = nullptr;
        cudaError_t r = cudaIpcOpenMemHandle(&ptr, h, cudaIpcMemLazyEnablePeerAccess);
        if (r != cudaSuccess) {
            (void)cudaGetLastError();
            return fail(LPP_ERR_CUDA, "cudaIpcOpenMemHandle for rank %d: %s", p, cudaGetErrorString(r));
        }
        e->peer_base[p] = (unsigned char*)ptr;
    }
    e->peer_ready = true;
    return LPP_OK;
}

// Test aid (not part of the public header): lets ONE rank of a tensor-parallel group run without its peers.
// Stores to the other ranks land in a private scratch buffer and nobody ever fills this rank's receive slots,
// so the first consuming GEMV's wait on its peers runs out after lpp_config.tp_wait_ms and the step ends
// with LPP_ERR_DEVICE_STATUS: the one way to see that path on a single GPU without a fault or a hang.
extern "C" lpp_status lpp_debug_tp_absent_peers(lpp_engine* e) {
    if (!e) return fail(LPP_ERR_INVALID_ARG, "null argument");
    if (!e->tp_buf || e->c.tp_size < 2) return fail(LPP_ERR_INVALID_ARG, "engine has no tensor-parallel exchange buffer");
    if (e->finalized) return fail(LPP_ERR_INVALID_ARG, "must precede lpp_finalize");
    CU(cudaSetDevice(e->c.device));
    if (!e->absent_peer) {
        CU(cudaMalloc(&e->absent_peer, e->tp_buf_bytes));
        CU(cudaMemset(e->absent_peer, 0, e->tp_buf_bytes));
    }
    for (int p = 0; p < e->c.tp_size; ++p)
        if (p != e->c.tp_rank && !e->peer_base[p]) e->peer_base[p] = e->absent_peer;
    e->peer_ready = true;
    return LPP_OK;
}

// Test aid (not part of the public header): one warp waits, with the engine's wait limit, on a shared-memory
// barrier that nothing ever arrives on.  The wait must run out, the kernel must return normally, and the
// call must fail with LPP_ERR_DEVICE_STATUS like a step whose copy never completed.
static __global__ void wait_probe_kernel(StepState* st) {
    __shared__ uint64_t bar;
    if (threadIdx.x == 0) {
        mbar_init(&bar, 1);
        mbar_fence_init();
    }
    __syncthreads();
    const bool ok = __all_sync(0xffffffffu, mbar_wait_bounded(&bar, 0u, st));
    if (!ok && threadIdx.x == 0) st->out_token = -2;
}
extern "C" lpp_status lpp_debug_wait_probe(lpp_engine* e) {
    NEED_READY(e);
    TRY(push_state(e, 0, 0, nullptr, nullptr, 0, 0.f, 0, 0));
    wait_probe_kernel<<<1, 32, 0, e->stream>>>(e->st);
    CU(cudaGetLastError());
    return pull_result(e, nullptr);
}

// Debugging aid (not part of the public header): per-CTA time stamps of the ring GEMV launches of one step.
extern "C" int lpp_debug_gemv_trace(lpp_engine* e, unsigned long long* out, int max_values) {
    if (!e || !e->gtrace || !out) return -1;
    const size_t n = (size_t)256 * e->num_sms * 8;
    if ((size_t)max_values < n) return -2;
    cudaStreamSynchronize(e->stream);
    if (cudaMemcpy(out, e->gtrace, n * sizeof(unsigned long long), cudaMemcpyDeviceToHost) != cudaSuccess) return -3;
    return e->num_sms;
}

// Debugging aid (not part of the public header): the exact sampler's entry lists of its last stage.
extern "C" int lpp_debug_sampler_entries(lpp_engine* e, int* counts, void* entries, float* scalars) {
    if (!e || !e->exact_sampler) return -1;
    cudaStreamSynchronize(e->stream);
    cudaMemcpy(counts, e->ex_entry_count, e->sample_blocks * sizeof(int), cudaMemcpyDeviceToHost);
    cudaMemcpy(entries, e->ex_entries, (size_t)e->sample_blocks * kExactMaxEntries * sizeof(ExactEntry), cudaMemcpyDeviceToHost);
    cudaMemcpy(scalars, e->ex_scalars, 64 * sizeof(float), cudaMemcpyDeviceToHost);
    return e->sample_blocks;
}

#ifdef LPP_TIMING_AIDS
extern "C" int lpp_debug_pf_trace(lpp_engine* e, unsigned long long* out) {
    if (!e) return -1;
    cudaStreamSynchronize(e->stream);
    return (int)cudaMemcpyFromSymbol(out, g_pf_trace, sizeof(unsigned long long) * 160 * 48);
}
#endif

extern "C" const char* lpp_strerror(int s) {
    switch (s) {
        case LPP_OK: return "ok";
        case LPP_ERR_INVALID_ARG: return "invalid argument";
        case LPP_ERR_CUDA: return "CUDA error";
        case LPP_ERR_NOT_READY: return "engine not ready";
        case LPP_ERR_NCCL: return "NCCL error";
        case LPP_ERR_DEVICE_STATUS: return "device reported an error status";
        case LPP_ERR_TOO_LARGE: return "request exceeds capacity";
        case LPP_ERR_NO_DEVICE: return "no usable CUDA device";
    }
    return "unknown status";
}
extern "C" const char* lpp_last_error(void) { return g_err.c_str(); }
extern "C" void* lpp_engine_stream(lpp_engine* e) { return e ? (void*)e->stream : nullptr; }
extern "C" int lpp_kernels_per_step(const lpp_engine* e) { return e ? e->kernels_full : 0; }

static void kind_bytes(const lpp_engine* e, int pos, int64_t* b) {
    const lpp_config& c = e->c;
    const int64_t D = c.dim, L = c.n_layers, V = c.vocab_size, esz = e->esz;
    for (int k = 0; k < kKinds; ++k) b[k] = 0;
    if (!e->layers.empty()) {
        for (const LayerRun& r : e->runs) {
            const ModelLayer& y = e->layers[r.layer];
            const lpp_layer_desc& d = y.d;
            const int64_t keys = d.window > 0 ? std::min<int64_t>(d.window, pos + 1) : pos + 1;
            const int64_t H = d.heads;
            if (d.mixer == LPP_MIXER_LATENT) {
                const int64_t row = d.kv_rank + d.rot_dim;
                b[kQkv] += (H * (d.dim + d.rot_dim) + row + H) * D * esz + 8 * D;
                b[kLatQuery] += H * d.dim * d.kv_rank * esz;
                b[kAttn] += (keys + 1) * row * e->kvesz;
                b[kLatValue] += H * d.vdim * d.kv_rank * esz;
                b[kOproj] += D * H * d.vdim * esz;
            } else if (d.mixer == LPP_MIXER_SHARED_KV) {
                b[kQkv] += ((1 + (d.gate ? 1 : 0)) * H + d.kv_heads) * d.dim * D * esz + 4 * D;
                b[kAttn] += (keys + 1) * d.kv_heads * (d.dim + d.rot_dims) * e->kvesz;
                b[kOproj] += D * H * d.dim * esz;
            } else {  // the recurrent state is read and written
                const int64_t E = d.inner, N = d.state;
                b[kQkv] += 2 * E * D * esz + 4 * D + E * (d.conv + 1 + d.conv) * 4;
                b[kScanIn] += (d.dt_rank + 2 * N) * E * esz;
                b[kScan] += E * d.dt_rank * esz + E * (3 * N + 2) * 4;
                b[kOproj] += D * E * esz;
            }
            if (d.ff > 0) {
                b[kGateUp] += (int64_t)2 * d.ff * D * esz + 8 * D;
                b[kDown] += D * d.ff * esz;
            }
        }
        b[kLmHead] = V * D * esz + 8 * D;
        return;
    }
    b[kQkv] = L * ((int64_t)(e->Dq + 2 * e->KVd) * D * esz + 4 * D) + 4 * D;  // + att norms + embedding row
    b[kAttn] = L * (int64_t)e->kvesz * 2 * e->KVd * ((int64_t)pos + 1) + L * (int64_t)e->kvesz * 2 * e->KVd;
    b[kOproj] = L * D * e->Dq * esz;
    b[kGateUp] = L * ((int64_t)2 * e->Fl * D * esz + 4 * D);
    b[kDown] = L * D * e->Fl * esz;
    b[kLmHead] = (tp_cls_sharded(e) ? V / c.tp_size : V) * D * esz + 4 * D;
}
extern "C" int64_t lpp_step_bytes(const lpp_engine* e, int pos) {
    if (!e) return 0;
    int64_t b[kKinds], t = 0;
    kind_bytes(e, pos, b);
    for (int k = 0; k < kKinds; ++k) t += b[k];
    return t;
}

// Average duration of one launch of `kind` when all of the step's launches of that kind run back to
// back, with the launch attributes the step uses (programmatic dependent launch between them) and one
// CUDA event pair on the engine stream around the whole sequence.  Every launch streams its own
// layer's weights, so consecutive launches never find them in L2.  Activations are whatever the
// buffers hold: the results are meaningless and the next real step overwrites them.
extern "C" lpp_status lpp_profile_kind(lpp_engine* e, int pos, int kind, int iters, float* ms_per_launch, int* launches) {
    NEED_READY(e);
    if (!ms_per_launch || !launches || iters <= 0 || kind < 0 || kind >= kKinds) return fail(LPP_ERR_INVALID_ARG, "bad argument");
    if (pos < 0 || pos >= e->c.seq_len) return fail(LPP_ERR_INVALID_ARG, "pos out of range");
    *ms_per_launch = 0.f;
    *launches = 0;
    if (e->recurrent) e->state_len = -1;
    lpp_sample_params sp = {0.8f, 1.1f};
    cudaGraphExec_t gx = nullptr;
    int n_kernels = 0;
    e->only_kind = kind;
    lpp_status rs = capture(e, true, false, &gx, &n_kernels);
    e->only_kind = -1;
    if (rs != LPP_OK) return rs;
    if (n_kernels == 0 && kind != kAllReduce) {
        cudaGraphExecDestroy(gx);
        return LPP_OK;
    }
    float total = 0.f;
    for (int it = 0; it < iters + 2 && rs == LPP_OK; ++it) {  // two warm-up rounds
        rs = push_state(e, 0, pos, &sp, nullptr, 0, 0.5f, 0, 0);
        if (rs != LPP_OK) break;
        cudaEventRecord(e->ev0, e->stream);
        cudaError_t le = cudaGraphLaunch(gx, e->stream);
        cudaEventRecord(e->ev1, e->stream);
        cudaError_t se = cudaStreamSynchronize(e->stream);
        if (le != cudaSuccess || se != cudaSuccess) {
            rs = fail(LPP_ERR_CUDA, "profile kind: %s", cudaGetErrorString(le != cudaSuccess ? le : se));
            break;
        }
        float t = 0.f;
        cudaEventElapsedTime(&t, e->ev0, e->ev1);
        if (it >= 2) total += t;
    }
    cudaGraphExecDestroy(gx);
    if (rs == LPP_OK) {
        *launches = n_kernels;
        *ms_per_launch = n_kernels > 0 ? total / iters / n_kernels : total / iters;
    }
    return rs;
}

extern "C" lpp_status lpp_profile_step(lpp_engine* e, int pos, int iters, const lpp_sample_params* spp, float* ms,
                                       int* launches, int64_t* bytes) {
    NEED_READY(e);
    if (!ms || !launches || !bytes || iters <= 0) return fail(LPP_ERR_INVALID_ARG, "bad argument");
    if (pos < 0 || pos >= e->c.seq_len) return fail(LPP_ERR_INVALID_ARG, "pos out of range");
    for (int k = 0; k < kKinds; ++k) ms[k] = 0.f, launches[k] = 0;
    kind_bytes(e, pos, bytes);
    if (e->recurrent) e->state_len = -1;
    // the sampler that is timed is the one the caller's workload runs (argmax and categorical paths differ)
    const lpp_sample_params sp = spp ? *spp : lpp_sample_params{0.f, 1.f};
    const int hist[3] = {1, 2, 3};
    // The step is captured once more with an event-record node before and after every kernel and
    // replayed as a graph, so the durations carry no host launch latency.  Event nodes sit between
    // the kernels, hence no programmatic overlap: these are isolated per-kernel times.
    cudaGraphExec_t gx = nullptr;
    lpp_status rs = LPP_OK;
    {
        cudaGraph_t g = nullptr;
        CU(cudaStreamBeginCapture(e->stream, cudaStreamCaptureModeThreadLocal));
        e->profiling = e->profiling_capture = true;
        Recorder R{e, e->stream};
        record_step(R, true);
        e->profiling = e->profiling_capture = false;
        cudaError_t ce = cudaStreamEndCapture(e->stream, &g);
        if (R.err != cudaSuccess || ce != cudaSuccess) {
            rs = fail(LPP_ERR_CUDA, "profile capture: %s", cudaGetErrorString(R.err != cudaSuccess ? R.err : ce));
        } else if (cudaGraphInstantiate(&gx, g, 0) != cudaSuccess) {
            rs = fail(LPP_ERR_CUDA, "profile graph instantiate failed");
        }
        if (g) cudaGraphDestroy(g);
        (void)cudaGetLastError();
    }
    for (int it = 0; it < iters + 1 && rs == LPP_OK; ++it) {  // iteration 0 is a warm-up
        rs = push_state(e, 0, pos, &sp, hist, 3, 0.5f, 0, 0);
        if (rs != LPP_OK) break;
        cudaError_t le = cudaGraphLaunch(gx, e->stream);
        cudaError_t se = cudaStreamSynchronize(e->stream);
        if (le != cudaSuccess || se != cudaSuccess) {
            rs = fail(LPP_ERR_CUDA, "profile step: %s", cudaGetErrorString(le != cudaSuccess ? le : se));
            break;
        }
        if (it == 0) continue;
        for (size_t i = 0; i + 1 < e->prof_events.size(); i += 2) {
            float t = 0.f;
            if (cudaEventElapsedTime(&t, e->prof_events[i], e->prof_events[i + 1]) != cudaSuccess) {
                rs = fail(LPP_ERR_CUDA, "cudaEventElapsedTime on graph event nodes failed");
                break;
            }
            ms[e->prof_kinds[i]] += t / iters;
            if (it == 1) launches[e->prof_kinds[i]]++;
        }
    }
    if (gx) cudaGraphExecDestroy(gx);
    for (cudaEvent_t ev : e->prof_events) cudaEventDestroy(ev);
    e->prof_events.clear();
    e->prof_kinds.clear();
    (void)cudaGetLastError();
    return rs;
}
