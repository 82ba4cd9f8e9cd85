// Maps through a narrow middle: y = f(W2 (W1 h)), W1 h being columns of a mixer's stacked projection (float32, possibly
// as split-K shares) and W2 [N, R] with R a few dozen.  One launch serves up to two such maps of the same rows, each
// with a function of its own behind it (the product never leaves the kernel unfinished):
//   FB_LR_PLAIN     y = z                                       z = W2 (W1 h) + bias   (bias [N], optional)
//   FB_LR_SIGMOID   y = 1 / (1 + exp(-z))
//   FB_LR_DECAY     y = exp(-exp(log_rate[c / group]) * log(1 + exp(z)))        (a decay per output, a rate per `group`
//                                                                                neighbouring outputs)
// y is float32 [rows, N].  What stands behind the product is float32 in both forms:
//   low_rank_mma   bfloat16 W2: tensor cores (mma.sync m16n8k16, float32 accumulation), a CTA of four warps takes 64 rows
//                  x 64 outputs; the middle is rounded once to bfloat16
//   low_rank_fma   any types: float32 multiply-adds, 32 rows x 64 outputs a CTA
#include "attention_common.cuh"
#include "rows.cuh"

namespace {

enum FbLowRank : int { FB_LR_PLAIN = 0, FB_LR_SIGMOID = 1, FB_LR_DECAY = 2 };

struct LowRankMap {
    const void* w;             // [N, R]
    int mid_off, R, N;         // the middle's columns in the projection rows, and the sizes
    int act;                   // an FbLowRank code
    const void* bias;          // [N] or nullptr
    const void* log_rate;      // [ceil(N / group)] for FB_LR_DECAY
    int group;
    float* out;                // [rows, N]
};
struct LowRankArgs {
    const float* proj; long proj_stride; int n_partials; long partial_stride;
    int n;
    LowRankMap map[2];
    int tiles_first;           // blockIdx.y below this: map[0]
};

template <typename TW>
__device__ __forceinline__ float lr_finish(const LowRankMap& m, float z, int c) {
    if (m.bias) z += fb_to_float(static_cast<const TW*>(m.bias)[c]);
    if (m.act == FB_LR_SIGMOID) return 1.0f / (1.0f + expf(-z));
    if (m.act == FB_LR_DECAY) {
        const float softplus = z > 20.0f ? z : log1pf(expf(z));
        return expf(-expf(fb_to_float(static_cast<const TW*>(m.log_rate)[c / m.group])) * softplus);
    }
    return z;
}

constexpr int LM_T = 64, LM_KC = 64, LM_LD = LM_KC + 8;

__global__ void __launch_bounds__(128)
low_rank_mma_kernel(const LowRankArgs a) {
    using bf16 = __nv_bfloat16;
    fb_pdl_launch_dependents();
    __shared__ __align__(16) bf16 As[LM_T][LM_LD];
    __shared__ __align__(16) bf16 Ws[LM_T][LM_LD];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const bool second = (int)blockIdx.y >= a.tiles_first;
    const LowRankMap m = second ? a.map[1] : a.map[0];
    const int m0 = blockIdx.x * LM_T, n0 = ((int)blockIdx.y - (second ? a.tiles_first : 0)) * LM_T;
    const bf16* w = static_cast<const bf16*>(m.w);
    const bool w_vec = m.R % 8 == 0 && (uintptr_t)w % 16 == 0;
    const bool a_vec = m.R % 4 == 0 && m.mid_off % 4 == 0 && a.proj_stride % 4 == 0 && a.partial_stride % 4 == 0 &&
                       (uintptr_t)a.proj % 16 == 0;
    float acc[LM_T / 8][4];
#pragma unroll
    for (int j = 0; j < LM_T / 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.0f;
    bool waited = false;
    for (int k0 = 0; k0 < m.R; k0 += LM_KC) {
        // the weights first: they are not of this step and need not wait for the kernel before
        if (w_vec) {
#pragma unroll
            for (int u = 0; u < LM_T * (LM_KC / 8) / 128; ++u) {
                const int idx = tid + 128 * u, nn = idx / (LM_KC / 8), k = (idx - nn * (LM_KC / 8)) * 8;
                uint4 raw = make_uint4(0u, 0u, 0u, 0u);
                if (n0 + nn < m.N && k0 + k < m.R) raw = *reinterpret_cast<const uint4*>(w + (size_t)(n0 + nn) * m.R + k0 + k);
                *reinterpret_cast<uint4*>(&Ws[nn][k]) = raw;
            }
        } else {
            for (int idx = tid; idx < LM_T * LM_KC; idx += 128) {
                const int nn = idx / LM_KC, k = idx - nn * LM_KC;
                Ws[nn][k] = (n0 + nn < m.N && k0 + k < m.R) ? w[(size_t)(n0 + nn) * m.R + k0 + k] : __float2bfloat16(0.0f);
            }
        }
        if (!waited) { fb_pdl_wait(); waited = true; }
        if (a_vec) {
#pragma unroll
            for (int u = 0; u < LM_T * (LM_KC / 4) / 128; ++u) {
                const int idx = tid + 128 * u, r = idx / (LM_KC / 4), k = (idx - r * (LM_KC / 4)) * 4;
                float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
                if (m0 + r < a.n && k0 + k < m.R)
                    v = slab_sum4(a.proj + (size_t)(m0 + r) * a.proj_stride + m.mid_off + k0 + k, a.n_partials, a.partial_stride);
                uint2 raw;
                raw.x = fb_attn::pack_bf16(v.x, v.y);
                raw.y = fb_attn::pack_bf16(v.z, v.w);
                *reinterpret_cast<uint2*>(&As[r][k]) = raw;
            }
        } else {
            for (int idx = tid; idx < LM_T * LM_KC; idx += 128) {
                const int r = idx / LM_KC, k = idx - r * LM_KC;
                float v = 0.0f;
                if (m0 + r < a.n && k0 + k < m.R)
                    v = fb_slab_sum(a.proj + (size_t)(m0 + r) * a.proj_stride, m.mid_off + k0 + k, a.n_partials, a.partial_stride);
                As[r][k] = __float2bfloat16(v);
            }
        }
        __syncthreads();
        if (m0 + warp * 16 < a.n) {
#pragma unroll
            for (int kk = 0; kk < LM_KC; kk += 16) {
                uint32_t af[4];
                af[0] = *reinterpret_cast<const uint32_t*>(&As[warp * 16 + g][kk + 2 * t]);
                af[1] = *reinterpret_cast<const uint32_t*>(&As[warp * 16 + g + 8][kk + 2 * t]);
                af[2] = *reinterpret_cast<const uint32_t*>(&As[warp * 16 + g][kk + 8 + 2 * t]);
                af[3] = *reinterpret_cast<const uint32_t*>(&As[warp * 16 + g + 8][kk + 8 + 2 * t]);
#pragma unroll
                for (int j = 0; j < LM_T / 8; ++j) {
                    const uint32_t b0 = *reinterpret_cast<const uint32_t*>(&Ws[j * 8 + g][kk + 2 * t]);
                    const uint32_t b1 = *reinterpret_cast<const uint32_t*>(&Ws[j * 8 + g][kk + 8 + 2 * t]);
                    fb_attn::mma_bf16(acc[j], af, b0, b1);
                }
            }
        }
        __syncthreads();
    }
    const bool pairs = m.N % 2 == 0 && (uintptr_t)m.out % 8 == 0;
#pragma unroll
    for (int j = 0; j < LM_T / 8; ++j)
#pragma unroll
        for (int hi = 0; hi < 2; ++hi) {
            const int r = m0 + warp * 16 + g + hi * 8, c = n0 + j * 8 + 2 * t;
            if (r >= a.n || c >= m.N) continue;
            float* dst = m.out + (size_t)r * m.N + c;
            const float y0 = lr_finish<bf16>(m, acc[j][2 * hi], c);
            if (c + 1 >= m.N) { dst[0] = y0; continue; }
            const float y1 = lr_finish<bf16>(m, acc[j][2 * hi + 1], c + 1);
            if (pairs) *reinterpret_cast<float2*>(dst) = make_float2(y0, y1);
            else { dst[0] = y0; dst[1] = y1; }
        }
}

constexpr int LF_TM = 32, LF_TN = 64, LF_KC = 16;

template <typename TW>
__global__ void __launch_bounds__(256)
low_rank_fma_kernel(const LowRankArgs a) {
    fb_pdl_launch_dependents();
    fb_pdl_wait();
    __shared__ float As[LF_KC][LF_TM + 1];
    __shared__ float Ws[LF_KC][LF_TN + 1];
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const bool second = (int)blockIdx.y >= a.tiles_first;
    const LowRankMap m = second ? a.map[1] : a.map[0];
    const int m0 = blockIdx.x * LF_TM, n0 = ((int)blockIdx.y - (second ? a.tiles_first : 0)) * LF_TN;
    const TW* w = static_cast<const TW*>(m.w);
    float acc[2][4] = {};
    for (int k0 = 0; k0 < m.R; k0 += LF_KC) {
        for (int idx = tid; idx < LF_TM * LF_KC; idx += 256) {
            const int r = idx / LF_KC, k = idx - r * LF_KC;
            As[k][r] = (m0 + r < a.n && k0 + k < m.R)
                ? fb_slab_sum(a.proj + (size_t)(m0 + r) * a.proj_stride, m.mid_off + k0 + k, a.n_partials, a.partial_stride) : 0.0f;
        }
        for (int idx = tid; idx < LF_TN * LF_KC; idx += 256) {
            const int nn = idx / LF_KC, k = idx - nn * LF_KC;
            Ws[k][nn] = (n0 + nn < m.N && k0 + k < m.R) ? fb_to_float(w[(size_t)(n0 + nn) * m.R + k0 + k]) : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < LF_KC; ++k)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                acc[0][i] = fmaf(As[k][ty], Ws[k][tx + 16 * i], acc[0][i]);
                acc[1][i] = fmaf(As[k][ty + 16], Ws[k][tx + 16 * i], acc[1][i]);
            }
        __syncthreads();
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int r = m0 + ty + 16 * j, c = n0 + tx + 16 * i;
            if (r < a.n && c < m.N) m.out[(size_t)r * m.N + c] = lr_finish<TW>(m, acc[j][i], c);
        }
}

}  // namespace

// Up to two maps of the same projection rows (count 1 or 2); the arrays hold one entry a map.  The weights, biases and
// rates of all maps share a dtype.
FB_API int fb_low_rank_maps(const float* proj, long long proj_stride, int n_partials, long long partial_stride, int n,
                            int count, const void* const* w, int w_dtype, const int* mid_off, const int* R, const int* N,
                            const int* act, const void* const* bias, const void* const* log_rate, const int* group,
                            float* const* out, cudaStream_t stream) {
    FB_REQUIRE(n >= 0 && (count == 1 || count == 2), "low_rank_maps: one or two maps wanted");
    LowRankArgs a = {};
    a.proj = proj; a.proj_stride = (long)proj_stride; a.n = n;
    a.n_partials = n_partials < 1 ? 1 : n_partials; a.partial_stride = (long)partial_stride;
    int tiles = 0;
    for (int i = 0; i < count; ++i) {
        FB_REQUIRE(w[i] && out[i] && R[i] > 0 && N[i] > 0 && mid_off[i] >= 0 && proj_stride >= (long long)mid_off[i] + R[i],
                   "low_rank_maps: bad sizes");
        FB_REQUIRE(act[i] >= FB_LR_PLAIN && act[i] <= FB_LR_DECAY, "low_rank_maps: unknown function %d", act[i]);
        FB_REQUIRE(act[i] != FB_LR_DECAY || (log_rate[i] && group[i] > 0), "low_rank_maps: a decay wants its rates");
        a.map[i] = {w[i], mid_off[i], R[i], N[i], act[i], bias[i], log_rate[i], group[i] > 0 ? group[i] : 1, out[i]};
        if (i == 0) a.tiles_first = (N[i] + LM_T - 1) / LM_T;
        tiles += (N[i] + LM_T - 1) / LM_T;
    }
    static_assert(LM_T == LF_TN, "both kernels tile the outputs alike");
    FB_REQUIRE(tiles <= 65535, "low_rank_maps: too many outputs");
    if (n == 0) return 0;
    if (w_dtype == FB_BF16) {
        fb_launch(low_rank_mma_kernel, dim3((n + LM_T - 1) / LM_T, tiles), dim3(128), 0, stream, a);
    } else {
        FB_REQUIRE(w_dtype == FB_F32, "low_rank_maps: unknown dtype code %d", w_dtype);
        fb_launch(low_rank_fma_kernel<float>, dim3((n + LF_TM - 1) / LF_TM, tiles), dim3(256), 0, stream, a);
    }
    return fb_check_launch("low_rank_maps");
}
