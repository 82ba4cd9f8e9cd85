// Shared vocabulary of the kernel library: dtype codes, typed loads and
// stores, the error channel, and warp/block reductions.
//
// Every exported launcher is `extern "C"`, takes raw device pointers, sizes
// and a stream, validates its arguments on the host, and returns 0 or a
// negative code after recording a message that `fb_last_error()` returns.
// The reference validates every launch the same way before it reaches the
// device (crates/forward/src/core/composites/standard_attn.rs:74-119).
#pragma once

#include <cuda_runtime.h>
#include <cuda_bf16.h>
#include <stdint.h>

#define FB_API extern "C" __attribute__((visibility("default")))

enum FbDtype : int { FB_F32 = 0, FB_BF16 = 1 };

// Status word bits that kernels may set (never trap, never spin forever).
enum FbStatus : int {
    FB_STATUS_BAD_TOKEN = 1,      // embedding id outside the table
    FB_STATUS_BAD_PAGE = 2,       // block table entry missing for a live key
    FB_STATUS_WAIT_TIMEOUT = 4,   // a bounded barrier wait ran out
};

int fb_fail(int code, const char* fmt, ...);   // records the message, returns code
int fb_check_launch(const char* what);          // cudaGetLastError -> fb_fail

#define FB_REQUIRE(cond, ...)                                   \
    do {                                                        \
        if (!(cond)) return fb_fail(-1, __VA_ARGS__);           \
    } while (0)

// ---- the device ---------------------------------------------------------------
constexpr int FB_MAX_DEVICES = 64;
int fb_device_ordinal();    // the current device, clamped into [0, FB_MAX_DEVICES)
int fb_sm_count();          // multiprocessors of the current device (asked once per device)

// Set-up that a launcher does once per device (raising a kernel's shared-memory limit): `flags` is the
// launcher's own static array of FB_MAX_DEVICES zeros.  Two host threads may both see "not yet" and both do the
// set-up, which is harmless because the set-up is idempotent.
inline bool fb_needs_setup(const bool* flags) { return !flags[fb_device_ordinal()]; }
inline void fb_setup_done(bool* flags) { flags[fb_device_ordinal()] = true; }

// Weights of the launchers' cost models (how many shares of K pay off): about what one device streams from
// memory and what one multiprocessor's tensor pipe multiplies.  They rank choices; nothing is sized by them.
constexpr double FB_MODEL_HBM_BYTES_PER_S = 6.0e12;
constexpr double FB_MODEL_SM_FLOPS = 9.0e12;

// ---- activations of gated feed-forwards -----------------------------------------
// out = act(gate) * up.  The code travels as a launcher argument (0 = no gating where that is an option).
// FB_ACT_LIMITED cuts both operands off and shifts the up side: with g = min(gate, limit) and u = up held to
// [-limit, limit], out = g sigmoid(slope g) (u + 1); `limit` and `slope` travel beside the code and mean nothing to the
// other activations.
enum FbAct : int { FB_ACT_SILU = 1, FB_ACT_GELU_TANH = 2, FB_ACT_LIMITED = 3 };
struct FbGate {
    int act;               // an FbAct code, 0: no gating
    float limit, slope;
};
inline bool fb_act_known(int act) { return act >= FB_ACT_SILU && act <= FB_ACT_LIMITED; }
inline bool fb_gate_known(const FbGate& gate) {
    return fb_act_known(gate.act) && (gate.act != FB_ACT_LIMITED || gate.limit > 0.0f);
}
__device__ __forceinline__ float fb_gelu_tanh(float z) {
    // 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3)))
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
__device__ __forceinline__ float fb_gate_times(const FbGate& gate, float g, float u) {
    if (gate.act == FB_ACT_LIMITED) {
        g = fminf(g, gate.limit);
        u = fminf(fmaxf(u, -gate.limit), gate.limit);
        return g / (1.0f + expf(-gate.slope * g)) * (u + 1.0f);
    }
    if (gate.act == FB_ACT_GELU_TANH) return fb_gelu_tanh(g) * u;
    return g / (1.0f + expf(-g)) * u;             // SiLU (crates/model-ops/src/ops/activation.rs:107-118)
}

// ---- activations that stand alone ---------------------------------------------
// out = act(z) for feed-forwards without a gate.  0 leaves z as it is.
enum FbPlainAct : int { FB_PLAIN_NONE = 0, FB_PLAIN_SILU = 1, FB_PLAIN_GELU_TANH = 2, FB_PLAIN_RELU_SQUARED = 3,
                        FB_PLAIN_GELU = 4 };
inline bool fb_plain_act_known(int act) { return act >= FB_PLAIN_NONE && act <= FB_PLAIN_GELU; }
__device__ __forceinline__ float fb_plain_act(int act, float z) {
    if (act == FB_PLAIN_RELU_SQUARED) { const float r = fmaxf(z, 0.0f); return r * r; }
    if (act == FB_PLAIN_SILU) return z / (1.0f + expf(-z));
    if (act == FB_PLAIN_GELU_TANH) return fb_gelu_tanh(z);
    if (act == FB_PLAIN_GELU) return 0.5f * z * (1.0f + erff(0.7071067811865476f * z));
    return z;
}

// ---- launches ---------------------------------------------------------------
// Kernels of a step run back to back on one stream.  With programmatic dependent launch the next kernel of the
// stream may be scheduled while this one is still draining: every kernel begins with fb_pdl_launch_dependents()
// (which lets the kernel after it start being placed once all of this kernel's blocks have begun) and calls
// fb_pdl_wait() before its first read of what the kernel before it produced and before its first global write.
// fb_pdl_wait() returns once all earlier kernels of the stream have completed and their writes are visible, so
// the order of results is that of ordinary stream launches; only launch latency and prologues overlap.
extern int g_fb_pdl;        // 1: launch with the programmatic-serialization attribute; 0: plain launches
// Kernel classes that are launched plainly even while programmatic dependent launch is on (a bit set of FbLaunchClass).
enum FbLaunchClass : int { FB_LAUNCH_OTHER = 0, FB_LAUNCH_GEMM_PAIR = 1, FB_LAUNCH_ATTENTION_TC = 2, FB_LAUNCH_GEMM_WIDE = 4 };
extern int g_fb_plain_classes;

__device__ __forceinline__ void fb_pdl_launch_dependents() {
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
}
__device__ __forceinline__ void fb_pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }

template <typename... KArgs, typename... Args>
inline void fb_launch_class(int launch_class, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem,
                            cudaStream_t stream, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[1];
    if (g_fb_pdl && !(launch_class & g_fb_plain_classes)) {
        attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[0].val.programmaticStreamSerializationAllowed = 1;
        cfg.attrs = attr;
        cfg.numAttrs = 1;
    }
    cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);     // an error shows in fb_check_launch()
}
template <typename... KArgs, typename... Args>
inline void fb_launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                      Args... args) {
    fb_launch_class(FB_LAUNCH_OTHER, kernel, grid, block, smem, stream, args...);
}

// ---- a running start for the product that follows ---------------------------
// The first `bytes` of every row of a weight matrix, fetched into L2 by a kernel that has the memory system to
// spare (the split-key attention kernel when its stream of cache ends), so that the product after it finds its
// first k-blocks there.  It travels in the launcher's arguments; a hint, nothing depends on it.
struct FbPrefetch {
    const char* base;      // nullptr: nothing to do
    int rows;
    long row_stride;       // bytes
    int bytes;             // per row, a multiple of 16
};
// The hint for `rows` rows `row_stride_bytes` apart from `base`, `bytes_per_row` of each; an empty hint when the
// arguments cannot be used (no base, unaligned rows, too few bytes).
FbPrefetch fb_make_prefetch(const void* base, long long rows, long long row_stride_bytes, int bytes_per_row);

__device__ __forceinline__ void fb_prefetch_issue(const FbPrefetch& pf, long worker, long n_workers) {
    if (!pf.base) return;
    for (long r = worker; r < pf.rows; r += n_workers)
        asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(pf.base + r * pf.row_stride), "r"(pf.bytes) : "memory");
}

// ---- block tables -------------------------------------------------------------
// The column of a request's table row that holds logical page `logical`.  The row's first `head` columns are the
// request's first `head` logical pages, which it keeps while it lives (the first keys under a window that keeps
// them visible; 0 as a rule); the columns behind them are its live pages from logical page `base` on.  Negative
// where the row has no column for the page (given back).
__host__ __device__ __forceinline__ int fb_table_column(int logical, int base, int head) {
    return logical < head ? logical : (logical >= base ? logical - base + head : -1);
}

// ---- which keys a query sees -----------------------------------------------------
// The first position that a query at position p sees under a window of the last `window` positions (0: none) and within
// its own chunk of `chunk` positions, counted from position 0 (0: no chunks).  It never falls as p grows.
__host__ __device__ __forceinline__ int fb_first_key(int p, int window, int chunk) {
    int first = window > 0 && p - window + 1 > 0 ? p - window + 1 : 0;
    if (chunk > 0) {
        const int start = p / chunk * chunk;
        if (start > first) first = start;
    }
    return first;
}

// ---- typed access -----------------------------------------------------------
__device__ __forceinline__ float fb_to_float(float v) { return v; }
__device__ __forceinline__ float fb_to_float(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T> __device__ __forceinline__ T fb_from_float(float v);
template <> __device__ __forceinline__ float fb_from_float<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 fb_from_float<__nv_bfloat16>(float v) {
    return __float2bfloat16_rn(v);
}

// ---- scores that pass a soft cap ---------------------------------------------------
// cap * tanh(y) with y = score / cap, for kernels whose scores are in units of their own (`cap` in the same).  For large
// |y| from one exponential, (1 - e) / (1 + e) with e = 2^(-2 log2(e) |y|); for small |y|, where 1 - e cancels, the Taylor
// series to y^7, whose next term is below 6e-8 of the result at the border.
__device__ __forceinline__ float fb_softcap(float y, float cap) {
    const float a = fabsf(y);
    const float e = exp2f(-2.8853900817779268f * a);
    const float big = __fdividef(1.0f - e, 1.0f + e);
    const float q = y * y;
    const float small = a * fmaf(q, fmaf(q, fmaf(q, -17.0f / 315.0f, 2.0f / 15.0f), -1.0f / 3.0f), 1.0f);
    return copysignf(cap * (a < 0.2f ? small : big), y);
}

// The same where the cap is at most FB_SOFTCAP_DIRECT (in base-2 units): cap (1 - 2 / (1 + 2^x)) with x = 2 log2(e) score /
// cap.  Its absolute error is about 2e-7 of the cap, which for caps of tens is far below what scores of 16-bit queries and
// keys carry; five instructions.
constexpr float FB_SOFTCAP_DIRECT = 400.0f;
__device__ __forceinline__ float fb_softcap_direct(float x, float cap) {
    float e, r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(x));
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.0f + e));       // (e = inf: 0; e = 0: 1)
    return fmaf(-2.0f * cap, r, cap);
}

// ---- reductions -------------------------------------------------------------
__device__ __forceinline__ float fb_warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float fb_warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// Block-wide sum; `scratch` holds at least 32 floats of shared memory.
// Every thread of the block must call it; every thread gets the result.
__device__ __forceinline__ float fb_block_sum(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int nwarps = (blockDim.x + 31) >> 5;
    v = fb_warp_sum(v);
    __syncthreads();                       // scratch may still be read from a previous call
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    float r = (lane < nwarps) ? scratch[lane] : 0.0f;
    r = fb_warp_sum(r);
    return r;
}
__device__ __forceinline__ float fb_block_max(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int nwarps = (blockDim.x + 31) >> 5;
    v = fb_warp_max(v);
    __syncthreads();
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    float r = (lane < nwarps) ? scratch[lane] : -INFINITY;
    r = fb_warp_max(r);
    return r;
}

// One number of a product that arrives as float32 split-K shares `partial_stride` apart: the shares are fetched eight
// at a time before any is added, so that their latencies overlap; the order of the additions is the plain one.
__device__ __forceinline__ float fb_slab_sum(const float* row, int c, int n_partials, long partial_stride) {
    float v = row[c];
    for (int p0 = 1; p0 < n_partials; p0 += 8) {
        float t[8];
#pragma unroll
        for (int u = 0; u < 8; ++u) t[u] = p0 + u < n_partials ? row[(size_t)(p0 + u) * partial_stride + c] : 0.0f;
#pragma unroll
        for (int u = 0; u < 8; ++u)
            if (p0 + u < n_partials) v += t[u];
    }
    return v;
}

// Dispatch a dtype code to a template parameter.
#define FB_DISPATCH_DTYPE(code, T, ...)                                   \
    do {                                                                  \
        if ((code) == FB_F32) { using T = float; __VA_ARGS__; }           \
        else if ((code) == FB_BF16) { using T = __nv_bfloat16; __VA_ARGS__; } \
        else return fb_fail(-1, "unknown dtype code %d", (int)(code));    \
    } while (0)
