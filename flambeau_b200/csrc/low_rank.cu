// Maps through a narrow middle: y = f(W2 (W1 h)), W1 h being columns of a mixer's stacked projection (float32, possibly
// as split-K shares) and W2 [N, R] with R a few dozen.  One launch serves up to two such maps of the same rows, each
// with a function of its own behind it (the product never leaves the kernel unfinished):
//   FB_LR_PLAIN     y = z                                       z = W2 (W1 h) + bias   (bias [N], optional)
//   FB_LR_SIGMOID   y = 1 / (1 + exp(-z))
//   FB_LR_DECAY     y = exp(-exp(log_rate[c / group]) * log(1 + exp(z)))        (a decay per output, a rate per `group`
//                                                                                neighbouring outputs)
// y is float32 [rows, N].  What stands behind the product is float32 in both forms:
//   low_rank_tiles, low_rank_mma   bfloat16 W2: tensor cores (mma.sync m16n8k16, float32 accumulation), a CTA of four warps
//                  takes 64 rows x 64 outputs (or several such tiles one after the other); the middle is rounded once to
//                  bfloat16
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

// The same for middles of up to LT_MAX_R columns whose weights can be fetched 16 bytes at a time: the rows' middles stay in
// shared memory for all NT output tiles of the CTA, whose weights arrive by asynchronous copies one tile ahead.
constexpr int LT_MAX_R = 256;
__host__ __device__ constexpr int lt_pitch(int R) { return (R + 15) / 16 * 16 + 8; }
inline size_t lt_smem(int R) { return (size_t)3 * LM_T * lt_pitch(R) * 2 + 4 * LM_T * sizeof(float); }

__device__ __forceinline__ float lr_finish_fast(int act, float z, float bias, float rate) {
    z += bias;
    if (act == FB_LR_SIGMOID) return __fdividef(1.0f, 1.0f + __expf(-z));
    if (act == FB_LR_DECAY) {
        // log(1 + exp(z)) = max(z, 0) + log(1 + e), e = exp(-|z|); for small e the series, where 1 + e would lose e's digits
        const float e = __expf(-fabsf(z));
        const float l = e < 0.02f ? e * fmaf(e, fmaf(e, fmaf(e, -0.25f, 1.0f / 3.0f), -0.5f), 1.0f) : __logf(1.0f + e);
        return expf(-rate * (fmaxf(z, 0.0f) + l));
    }
    return z;
}

template <int NT>
__global__ void __launch_bounds__(128)
low_rank_tiles_kernel(const LowRankArgs a) {
    using bf16 = __nv_bfloat16;
    fb_pdl_launch_dependents();
    extern __shared__ __align__(16) unsigned char lt_raw[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const bool second = (int)blockIdx.y >= a.tiles_first;
    const LowRankMap m = second ? a.map[1] : a.map[0];
    const int m0 = blockIdx.x * LM_T, tile0 = ((int)blockIdx.y - (second ? a.tiles_first : 0)) * NT;
    const int tiles = min(NT, (m.N + LM_T - 1) / LM_T - tile0);
    const int P = lt_pitch(m.R), K = P - 8;
    bf16* As = reinterpret_cast<bf16*>(lt_raw);                       // [64][P]
    bf16* Ws = As + LM_T * P;                                         // [2][64][P]
    float* col = reinterpret_cast<float*>(Ws + 2 * LM_T * P);         // [2][bias: 64 | rate: 64]
    const bf16* w = static_cast<const bf16*>(m.w);
    auto fetch = [&](int tile) {
        bf16* dst = Ws + (tile & 1) * LM_T * P;
        const int n0 = (tile0 + tile) * LM_T, chunks = K / 8;
        for (int idx = tid; idx < LM_T * chunks; idx += 128) {
            const int r = idx / chunks, k = (idx - r * chunks) * 8;
            if (n0 + r < m.N && k < m.R)
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst + r * P + k)),
                             "l"(w + (size_t)(n0 + r) * m.R + k) : "memory");
            else
                *reinterpret_cast<uint4*>(dst + r * P + k) = make_uint4(0u, 0u, 0u, 0u);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        if (tid < LM_T && n0 + tid < m.N) {
            float* c = col + (tile & 1) * 2 * LM_T + tid;
            c[0] = m.bias ? fb_to_float(static_cast<const bf16*>(m.bias)[n0 + tid]) : 0.0f;
            c[LM_T] = m.act == FB_LR_DECAY ? expf(fb_to_float(static_cast<const bf16*>(m.log_rate)[(n0 + tid) / m.group])) : 0.0f;
        }
    };
    fetch(0);                                          // (not of this step: it need not wait for the kernel before)
    fb_pdl_wait();
    const bool a_vec = m.mid_off % 4 == 0 && a.proj_stride % 4 == 0 && a.partial_stride % 4 == 0 && (uintptr_t)a.proj % 16 == 0;
    const int quads = K / 4;
#pragma unroll 4
    for (int idx = tid; idx < LM_T * quads; idx += 128) {
        const int r = idx / quads, k = (idx - r * quads) * 4;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (m0 + r < a.n && k < m.R) {
            const float* src = a.proj + (size_t)(m0 + r) * a.proj_stride + m.mid_off + k;
            if (a_vec) {
                v = slab_sum4(src, a.n_partials, a.partial_stride);
            } else {
                v.x = fb_slab_sum(src, 0, a.n_partials, a.partial_stride); v.y = fb_slab_sum(src, 1, a.n_partials, a.partial_stride);
                v.z = fb_slab_sum(src, 2, a.n_partials, a.partial_stride); v.w = fb_slab_sum(src, 3, a.n_partials, a.partial_stride);
            }
        }
        uint2 raw;
        raw.x = fb_attn::pack_bf16(v.x, v.y);
        raw.y = fb_attn::pack_bf16(v.z, v.w);
        *reinterpret_cast<uint2*>(As + r * P + k) = raw;
    }
    const bool pairs = m.N % 2 == 0 && (uintptr_t)m.out % 8 == 0;
    for (int tile = 0; tile < tiles; ++tile) {
        if (tile + 1 < tiles) {
            fetch(tile + 1);                           // (its buffer's last readers passed the barrier at the loop's end)
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const int n0 = (tile0 + tile) * LM_T;
        if (m0 + warp * 16 < a.n) {                    // (warp-uniform)
            float acc[LM_T / 8][4];
#pragma unroll
            for (int j = 0; j < LM_T / 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.0f;
            const bf16* ar = As + (warp * 16 + g) * P + 2 * t;
            const bf16* wr = Ws + (tile & 1) * LM_T * P + g * P + 2 * t;
            for (int kk = 0; kk < K; kk += 16) {
                uint32_t af[4];
                af[0] = *reinterpret_cast<const uint32_t*>(ar + kk);
                af[1] = *reinterpret_cast<const uint32_t*>(ar + 8 * P + kk);
                af[2] = *reinterpret_cast<const uint32_t*>(ar + kk + 8);
                af[3] = *reinterpret_cast<const uint32_t*>(ar + 8 * P + kk + 8);
#pragma unroll
                for (int j = 0; j < LM_T / 8; ++j)
                    fb_attn::mma_bf16(acc[j], af, *reinterpret_cast<const uint32_t*>(wr + j * 8 * P + kk),
                                      *reinterpret_cast<const uint32_t*>(wr + j * 8 * P + kk + 8));
            }
            const float* c0 = col + (tile & 1) * 2 * LM_T;
#pragma unroll
            for (int j = 0; j < LM_T / 8; ++j) {
                const int cc = j * 8 + 2 * t, c = n0 + cc;
                const float b0 = c0[cc], b1 = c0[cc + 1], r0 = c0[LM_T + cc], r1 = c0[LM_T + cc + 1];
#pragma unroll
                for (int hi = 0; hi < 2; ++hi) {
                    const int r = m0 + warp * 16 + g + hi * 8;
                    if (r >= a.n || c >= m.N) continue;
                    float* dst = m.out + (size_t)r * m.N + c;
                    const float y0 = lr_finish_fast(m.act, acc[j][2 * hi], b0, r0), y1 = lr_finish_fast(m.act, acc[j][2 * hi + 1], b1, r1);
                    if (pairs) { *reinterpret_cast<float2*>(dst) = make_float2(y0, y1); continue; }
                    dst[0] = y0;
                    if (c + 1 < m.N) dst[1] = y1;
                }
            }
        }
        __syncthreads();
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
        bool resident = true;
        int widest = 0;
        for (int i = 0; i < count; ++i) {
            resident = resident && R[i] % 8 == 0 && R[i] <= LT_MAX_R && (uintptr_t)w[i] % 16 == 0;
            widest = R[i] > widest ? R[i] : widest;
        }
        if (resident) {
            const int NT = n > 64 ? 4 : 1;             // (few rows: the tiles spread over the device)
            auto groups = [&](int i) { return ((N[i] + LM_T - 1) / LM_T + NT - 1) / NT; };
            a.tiles_first = groups(0);
            const dim3 grid((n + LM_T - 1) / LM_T, groups(0) + (count > 1 ? groups(1) : 0));
            auto kernel = NT == 4 ? low_rank_tiles_kernel<4> : low_rank_tiles_kernel<1>;
            const size_t smem = lt_smem(widest);
            if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            fb_launch(kernel, grid, dim3(128), smem, stream, a);
            return fb_check_launch("low_rank_maps");
        }
        fb_launch(low_rank_mma_kernel, dim3((n + LM_T - 1) / LM_T, tiles), dim3(128), 0, stream, a);
    } else {
        FB_REQUIRE(w_dtype == FB_F32, "low_rank_maps: unknown dtype code %d", w_dtype);
        fb_launch(low_rank_fma_kernel<float>, dim3((n + LF_TM - 1) / LF_TM, tiles), dim3(256), 0, stream, a);
    }
    return fb_check_launch("low_rank_maps");
}
