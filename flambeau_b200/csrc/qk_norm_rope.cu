// What lies between a fused q/k/v projection and the attention when queries and keys pass an RMS norm on the way:
// add the projection's split-K shares, normalise q and k, rotate them, round q once, and put k and v into their
// cache pages.  One CTA per token; the row's q and k live in shared memory between the two passes.
//
// The norm's reach is an argument: over every head alone (FB_QK_NORM_HEAD: width = head size, one weight of
// that size shared by the heads) or over the whole projection at once (FB_QK_NORM_PROJECTION: width = heads * head
// size, a weight of that size), before the rotation in both cases.  The weight enters as (w + weight_offset).
// Rotation: the first 2 * half dimensions of a head, dimension i paired with i + half, angles from the step's
// cos/sin tables [n, half]; the rest of the head passes unchanged.  Value rows have a width of their own, and their
// columns may be the keys' (`v_off`): the values are then the keys as projected, before norm and rotation.  A bias over
// the q, k and v columns (optional) joins the projection first.  `maps` neighbouring heads of q and of k may belong to
// one head with several score maps: each is normalised and rotated alone, and a key's maps lie side by side in the
// cache, whose key/value heads are then nkv / maps.
//
// Heads that are normalised alone (or not at all) and whose sizes are multiples of 4 go to a second kernel, one warp a
// head: shares fetched 16 bytes at a time, the norm within the warp, the pairs exchanged through the warp's own stretch
// of shared memory.
#include "rows.cuh"

enum FbQkNorm : int { FB_QK_NORM_NONE = 0, FB_QK_NORM_HEAD = 1, FB_QK_NORM_PROJECTION = 2 };

__device__ __forceinline__ float qkr_slab_sum(const float* row, int c, int n_partials, long partial_stride) {
    float v = row[c];
    for (int p = 1; p < n_partials; ++p) v += row[(size_t)p * partial_stride + c];
    return v;
}

template <typename TW, typename T>
__global__ void __launch_bounds__(1024)
qk_norm_rope_kv_write_kernel(const float* __restrict__ proj, long proj_stride, int n_partials, long partial_stride,
                             const TW* __restrict__ bias, const TW* __restrict__ q_weight,
                             const TW* __restrict__ k_weight, int scope, float eps, float weight_offset, const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                             int half, T* __restrict__ q_out, long q_out_stride, const int* __restrict__ positions,
                             const int* __restrict__ row_seq, const int* __restrict__ block_table, int table_stride,
                             const int* __restrict__ table_base, int table_head, T* __restrict__ k_pool,
                             T* __restrict__ v_pool, int page_size, int n_pages, int nh, int nkv, int maps, int hd,
                             int vd, int v_off, int write_kv, int* status) {
    fb_pdl_launch_dependents();
    fb_pdl_wait();
    extern __shared__ float sh[];                      // [qw + kw] the row's q and k; then one factor per head
    __shared__ float red[32];
    const int row = blockIdx.x, tid = threadIdx.x;
    const int nv = nkv / maps;                         // key/value heads of the cache
    const int qw = nh * hd, kw = nkv * hd, vw = nv * vd;
    const int heads = nh + nkv;
    float* inv = sh + qw + kw;                         // [heads]
    const float* pr = proj + (size_t)row * proj_stride;
    for (int c = tid; c < qw + kw; c += blockDim.x)
        sh[c] = qkr_slab_sum(pr, c, n_partials, partial_stride) + (bias ? fb_to_float(bias[c]) : 0.0f);
    __syncthreads();
    if (scope == FB_QK_NORM_PROJECTION) {
        float sq = 0.0f, sk = 0.0f;
        for (int c = tid; c < qw; c += blockDim.x) sq = fmaf(sh[c], sh[c], sq);
        for (int c = tid; c < kw; c += blockDim.x) sk = fmaf(sh[qw + c], sh[qw + c], sk);
        sq = fb_block_sum(sq, red);
        sk = fb_block_sum(sk, red);
        const float iq = 1.0f / sqrtf(sq / (float)qw + eps), ik = 1.0f / sqrtf(sk / (float)kw + eps);
        for (int h = tid; h < heads; h += blockDim.x) inv[h] = h < nh ? iq : ik;
    } else if (scope == FB_QK_NORM_HEAD) {
        const int warp = tid >> 5, lane = tid & 31, nwarps = blockDim.x >> 5;
        for (int h = warp; h < heads; h += nwarps) {
            const float* x = sh + (size_t)h * hd;
            float s = 0.0f;
            for (int d = lane; d < hd; d += 32) s = fmaf(x[d], x[d], s);
            s = fb_warp_sum(s);
            if (lane == 0) inv[h] = 1.0f / sqrtf(s / (float)hd + eps);
        }
    } else {
        for (int h = tid; h < heads; h += blockDim.x) inv[h] = 1.0f;
    }
    __syncthreads();

    // where this token's key and value rows go
    T* k_dst = nullptr;
    T* v_dst = nullptr;
    if (write_kv) {
        const int p = positions[row], seq = row_seq[row];
        const int entry = fb_table_column(p / page_size, table_base ? table_base[seq] : 0, table_head);
        const int page = (entry >= 0 && entry < table_stride) ? block_table[(size_t)seq * table_stride + entry] : -1;
        if (page < 0 || page >= n_pages) {
            if (tid == 0) atomicOr(status, FB_STATUS_BAD_PAGE);
        } else {
            // pools are [page][kv head][slot][row]: head g's row of this token
            k_dst = k_pool + ((size_t)page * nv * page_size + (p % page_size)) * maps * hd;
            v_dst = v_pool + ((size_t)page * nv * page_size + (p % page_size)) * vd;
        }
    }
    const float* cs = half ? cos_t + (size_t)row * half : nullptr;
    const float* sn = half ? sin_t + (size_t)row * half : nullptr;
    const int n_items = write_kv ? heads * hd : qw;
    for (int e = tid; e < n_items; e += blockDim.x) {
        const int h = e / hd, d = e - h * hd;
        const bool is_q = h < nh;
        const TW* w = is_q ? q_weight : k_weight;
        // the weight's index: within the whole projection, or within the head
        const int wbase = scope == FB_QK_NORM_PROJECTION ? (is_q ? h : h - nh) * hd : 0;
        const float f = inv[h];
        auto val = [&](int dd) -> float {
            const float x = sh[(size_t)h * hd + dd] * f;
            return (w && scope != FB_QK_NORM_NONE) ? x * (fb_to_float(w[wbase + dd]) + weight_offset) : x;
        };
        float y;
        if (d < half) {
            y = val(d) * cs[d] - val(d + half) * sn[d];
        } else if (d < 2 * half) {
            y = val(d) * cs[d - half] + val(d - half) * sn[d - half];
        } else {
            y = val(d);
        }
        if (is_q) {
            q_out[(size_t)row * q_out_stride + e] = fb_from_float<T>(y);
        } else if (k_dst) {
            const int g = (h - nh) / maps, map = (h - nh) - g * maps;
            k_dst[((size_t)g * page_size * maps + map) * hd + d] = fb_from_float<T>(y);
        }
    }
    if (v_dst) {
        for (int e = tid; e < vw; e += blockDim.x) {
            const int g = e / vd, d = e - g * vd;
            v_dst[(size_t)g * page_size * vd + d] =
                fb_from_float<T>(qkr_slab_sum(pr, v_off + e, n_partials, partial_stride) +
                                 (bias ? fb_to_float(bias[v_off + e]) : 0.0f));
        }
    }
}

// A warp takes HPW neighbouring heads of a row: heads 0 .. nh - 1 are queries, the nkv behind them keys, the nkv / maps
// behind those values (none where the values are the keys as projected: the key's warp then writes both).  NV = float4 a lane
// holds of a head.  Every load of the warp's heads is issued before the first use.  The two members of a rotated pair lie
// 2 * half / 8 lanes apart where NV is 1 and half a multiple of 4 (one exchange between lanes); otherwise they meet in the
// warp's stretch of shared memory.
constexpr int QKR_WARPS = 8;
template <typename TW, typename T, int NV, int HPW>
__global__ void __launch_bounds__(32 * QKR_WARPS)
qk_norm_rope_heads_kernel(const float* __restrict__ proj, long proj_stride, int n_partials, long partial_stride,
                          const TW* __restrict__ bias, const TW* __restrict__ q_weight,
                          const TW* __restrict__ k_weight, float eps, float weight_offset, const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                          int half, T* __restrict__ q_out, long q_out_stride, const int* __restrict__ positions,
                          const int* __restrict__ row_seq, const int* __restrict__ block_table, int table_stride,
                          const int* __restrict__ table_base, int table_head, T* __restrict__ k_pool,
                          T* __restrict__ v_pool, int page_size, int n_pages, int n, int nh, int nkv, int maps, int hd,
                          int vd, int v_off, int v_is_k, int write_kv, int* status) {
    fb_pdl_launch_dependents();
    extern __shared__ float sh[];                      // [QKR_WARPS][hd], where pairs meet in shared memory
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int nv = nkv / maps;                         // key/value heads of the cache
    const int per_row = nh + (write_kv ? (v_is_k ? nkv : nkv + nv) : 0);
    const int groups = (per_row + HPW - 1) / HPW;
    const long item = (long)blockIdx.x * QKR_WARPS + warp;
    const int row = (int)(item / groups), h0 = (int)(item - (long)row * groups) * HPW;
    const bool by_lanes = NV == 1 && (half & 3) == 0;
    float4 wq[NV], wk[NV];                             // the norms' weights (parameters, not of this step)
    if (q_weight) {
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = lane + 32 * i;
            wq[i] = wk[i] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (c >= hd >> 2) continue;
            wq[i] = Vec4<TW>::load(q_weight + 4 * c);
            wk[i] = Vec4<TW>::load(k_weight + 4 * c);
            wq[i].x += weight_offset; wq[i].y += weight_offset; wq[i].z += weight_offset; wq[i].w += weight_offset;
            wk[i].x += weight_offset; wk[i].y += weight_offset; wk[i].z += weight_offset; wk[i].w += weight_offset;
        }
    }
    fb_pdl_wait();
    if (row >= n) return;
    float4 x[HPW][NV];
#pragma unroll
    for (int j = 0; j < HPW; ++j) {
        const int h = h0 + j;
        const bool is_v = h >= nh + nkv;
        const int nvec = (is_v ? vd : hd) >> 2;
        const float* src = proj + (size_t)row * proj_stride +
                           (is_v ? (size_t)v_off + (size_t)(h - nh - nkv) * vd : (size_t)h * hd);
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = lane + 32 * i;
            x[j][i] = h < per_row && c < nvec ? Vec4<float>::load(src + 4 * c) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    }
    // the pairs' cosines and sines: this lane's four columns are four pairs, first members for columns below `half`
    float4 cs = make_float4(0.f, 0.f, 0.f, 0.f), sn = cs;
    const bool turns = by_lanes && 4 * lane < 2 * half, second = 4 * lane >= half;
    if (turns) {
        const size_t at = (size_t)row * half + 4 * lane - (second ? half : 0);
        cs = Vec4<float>::load(cos_t + at);
        sn = Vec4<float>::load(sin_t + at);
        if (!second) { sn.x = -sn.x; sn.y = -sn.y; sn.z = -sn.z; sn.w = -sn.w; }
    }
    size_t cache_row = 0;                              // + head * page_size: the token's row in a pool
    bool cached = false;
    if (h0 + HPW > nh && write_kv) {
        const int p = positions[row], seq = row_seq[row];
        const int entry = fb_table_column(p / page_size, table_base ? table_base[seq] : 0, table_head);
        const int page = (entry >= 0 && entry < table_stride) ? block_table[(size_t)seq * table_stride + entry] : -1;
        cached = page >= 0 && page < n_pages;
        if (!cached && lane == 0) atomicOr(status, FB_STATUS_BAD_PAGE);
        cache_row = (size_t)page * nv * page_size + (p % page_size);
    }
    if (bias) {
#pragma unroll
        for (int j = 0; j < HPW; ++j) {
            const int h = h0 + j;
            const bool is_v = h >= nh + nkv;
            const int nvec = (is_v ? vd : hd) >> 2;
            const TW* src = bias + (is_v ? v_off + (h - nh - nkv) * vd : h * hd);
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const int c = lane + 32 * i;
                if (h >= per_row || c >= nvec) continue;
                const float4 b = Vec4<TW>::load(src + 4 * c);
                x[j][i].x += b.x; x[j][i].y += b.y; x[j][i].z += b.z; x[j][i].w += b.w;
            }
        }
    }
    if (n_partials > 1) {
        // one head: its shares eight at a time; several: share after share, a load of every head in flight
        for (int p0 = 1; p0 < n_partials; p0 += HPW == 1 ? n_partials - 1 : 1) {
#pragma unroll
            for (int j = 0; j < HPW; ++j) {
                const int h = h0 + j;
                const bool is_v = h >= nh + nkv;
                const int nvec = (is_v ? vd : hd) >> 2;
                const float* src = proj + (size_t)row * proj_stride + (size_t)p0 * partial_stride +
                                   (is_v ? (size_t)v_off + (size_t)(h - nh - nkv) * vd : (size_t)h * hd);
#pragma unroll
                for (int i = 0; i < NV; ++i) {
                    const int c = lane + 32 * i;
                    if (h >= per_row || c >= nvec) continue;
                    const float4 more = HPW == 1 ? slab_sum4(src + 4 * c, n_partials - 1, partial_stride)
                                                 : Vec4<float>::load(src + 4 * c);
                    x[j][i].x += more.x; x[j][i].y += more.y; x[j][i].z += more.z; x[j][i].w += more.w;
                }
            }
        }
    }
#pragma unroll
    for (int j = 0; j < HPW; ++j) {
        const int h = h0 + j;
        if (h >= per_row) break;
        const bool is_q = h < nh, is_v = h >= nh + nkv;
        const int g = is_q ? h : is_v ? h - nh - nkv : h - nh;
        const int nvec = (is_v ? vd : hd) >> 2;
        if (!is_q && !cached) continue;
        // the token's row in a pool (a key's maps share one)
        const size_t at = is_q ? 0 : cache_row + (size_t)(is_v ? g : g / maps) * page_size;
        if (is_v || (!is_q && v_is_k)) {
            T* v_dst = v_pool + at * vd;
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const int c = lane + 32 * i;
                if (c < nvec) Vec4<T>::store(v_dst + 4 * c, x[j][i]);
            }
            if (is_v) continue;
        }
        if (q_weight) {
            float s = 0.0f;
#pragma unroll
            for (int i = 0; i < NV; ++i)
                s += x[j][i].x * x[j][i].x + x[j][i].y * x[j][i].y + x[j][i].z * x[j][i].z + x[j][i].w * x[j][i].w;
            const float f = 1.0f / sqrtf(fb_warp_sum(s) / (float)hd + eps);
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const float4 w = is_q ? wq[i] : wk[i];
                x[j][i].x *= f * w.x; x[j][i].y *= f * w.y; x[j][i].z *= f * w.z; x[j][i].w *= f * w.w;
            }
        }
        if (by_lanes) {
            if (half > 0) {
                const int mate = (second ? lane - (half >> 2) : lane + (half >> 2)) & 31;
                float4 o;
                o.x = __shfl_sync(0xffffffffu, x[j][0].x, mate); o.y = __shfl_sync(0xffffffffu, x[j][0].y, mate);
                o.z = __shfl_sync(0xffffffffu, x[j][0].z, mate); o.w = __shfl_sync(0xffffffffu, x[j][0].w, mate);
                if (turns) {
                    x[j][0].x = x[j][0].x * cs.x + o.x * sn.x; x[j][0].y = x[j][0].y * cs.y + o.y * sn.y;
                    x[j][0].z = x[j][0].z * cs.z + o.z * sn.z; x[j][0].w = x[j][0].w * cs.w + o.w * sn.w;
                }
            }
        } else if (half > 0) {
            float* mine = sh + (size_t)warp * hd;
            __syncwarp();                              // (the head before has been read)
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const int c = lane + 32 * i;
                if (c < nvec && 4 * c < 2 * half) Vec4<float>::store(mine + 4 * c, x[j][i]);
            }
            __syncwarp();
            const float* ct = cos_t + (size_t)row * half;
            const float* st = sin_t + (size_t)row * half;
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const int d0 = 4 * (lane + 32 * i);
                if (d0 >= 2 * half) continue;
                float* xe = reinterpret_cast<float*>(&x[j][i]);
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int d = d0 + e;
                    if (d < half) xe[e] = xe[e] * ct[d] - mine[d + half] * st[d];
                    else if (d < 2 * half) xe[e] = xe[e] * ct[d - half] + mine[d - half] * st[d - half];
                }
            }
        }
        T* dst = is_q ? q_out + (size_t)row * q_out_stride + (size_t)h * hd : k_pool + (at * maps + g % maps) * hd;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = lane + 32 * i;
            if (c < nvec) Vec4<T>::store(dst + 4 * c, x[j][i]);
        }
    }
}

// proj: float32 rows [q: nh*hd | k: nkv*hd | ... v: nkv/maps*vd from column v_off on ...], possibly as n_partials shares
// partial_stride elements apart.  bias (may be null): dtype w_dtype, by the same columns.  Pools: keys [page][nkv / maps]
// [slot][maps * hd], values [page][nkv / maps][slot][vd].
// q_weight / k_weight (dtype w_dtype): [hd] each for FB_QK_NORM_HEAD, [nh*hd] and [nkv*hd] for FB_QK_NORM_PROJECTION.
FB_API int fb_qk_norm_rope_kv_write(const float* proj, long long proj_stride, int n_partials, long long partial_stride,
                                    const void* bias, const void* q_weight, const void* k_weight, int w_dtype, int scope, float eps,
                                    float weight_offset, const float* cos_t, const float* sin_t, int half, void* q_out,
                                    long long q_out_stride, int out_dtype, const int* positions, const int* row_seq,
                                    const int* block_table, int table_stride, const int* table_base, int table_head,
                                    void* k_pool, void* v_pool, int page_size, int n_pages, int n, int nh, int nkv, int maps, int hd, int vd,
                                    int v_off, int write_kv, int* status, cudaStream_t stream) {
    FB_REQUIRE(n >= 0 && nh > 0 && nkv > 0 && hd > 0 && vd > 0, "qk_norm_rope_kv_write: bad sizes");
    FB_REQUIRE(scope >= FB_QK_NORM_NONE && scope <= FB_QK_NORM_PROJECTION, "qk_norm_rope_kv_write: unknown reach %d", scope);
    FB_REQUIRE(half >= 0 && 2 * half <= hd, "qk_norm_rope_kv_write: rotary width %d exceeds head size %d", 2 * half, hd);
    FB_REQUIRE(half == 0 || (cos_t && sin_t), "qk_norm_rope_kv_write: rotary tables missing");
    FB_REQUIRE(!write_kv || (positions && row_seq && block_table && k_pool && v_pool && page_size > 0 && n_pages > 0),
               "qk_norm_rope_kv_write: cache arguments missing");
    const int k_off = nh * hd;
    FB_REQUIRE(v_off >= k_off && (v_off != k_off || vd == hd), "qk_norm_rope_kv_write: values that are the keys have their size");
    FB_REQUIRE(maps >= 1 && nkv % maps == 0 && (maps == 1 || v_off != k_off),
               "qk_norm_rope_kv_write: %d key heads in maps of %d", nkv, maps);
    const int nv = nkv / maps;
    FB_REQUIRE(proj_stride >= (long long)(nh + nkv) * hd && proj_stride >= (long long)v_off + (long long)nv * vd,
               "qk_norm_rope_kv_write: projection rows are too short");
    if (n == 0) return 0;
    if (n_partials < 1) n_partials = 1;
    const size_t esize = out_dtype == FB_BF16 ? 2 : 4;
    const size_t wsize = w_dtype == FB_BF16 ? 2 : 4;
    auto aligned = [](const void* p, size_t to) { return (uintptr_t)p % to == 0; };
    if (scope != FB_QK_NORM_PROJECTION && hd % 4 == 0 && vd % 4 == 0 && hd <= 512 && vd <= 512 && v_off % 4 == 0 &&
        proj_stride % 4 == 0 && partial_stride % 4 == 0 && q_out_stride % 4 == 0 && aligned(proj, 16) &&
        aligned(q_out, 4 * esize) && aligned(k_pool, 4 * esize) && aligned(v_pool, 4 * esize) &&
        aligned(q_weight, 4 * wsize) && aligned(k_weight, 4 * wsize) && aligned(bias, 4 * wsize)) {
        if (scope == FB_QK_NORM_NONE) q_weight = k_weight = nullptr;
        const int v_is_k = v_off == k_off ? 1 : 0;
        // (a few rows: one head a warp, so that the heads spread over the device; a portion: four, for loads in flight)
        const int hpw = n <= 64 ? 1 : 4;
        const int per_row = nh + (write_kv ? (v_is_k ? nkv : nkv + nv) : 0);
        const long items = (long)n * ((per_row + hpw - 1) / hpw);
        const unsigned blocks = (unsigned)((items + QKR_WARPS - 1) / QKR_WARPS);
        const size_t smem_h = (size_t)QKR_WARPS * hd * sizeof(float);
        const int widest = hd > vd ? hd : vd;
#define FB_QKR_HEADS(NV_, HPW_)                                                                                       \
        FB_DISPATCH_DTYPE(w_dtype, TW, FB_DISPATCH_DTYPE(out_dtype, T,                                                \
            (fb_launch((qk_norm_rope_heads_kernel<TW, T, NV_, HPW_>), dim3(blocks), dim3(32 * QKR_WARPS), smem_h, stream, \
                       proj, (long)proj_stride, n_partials, (long)partial_stride, (const TW*)bias, (const TW*)q_weight, (const TW*)k_weight, \
                       eps, weight_offset, cos_t, sin_t, half, (T*)q_out, (long)q_out_stride, positions, row_seq, block_table, \
                       table_stride, table_base, table_head, (T*)k_pool, (T*)v_pool, page_size, n_pages, n, nh, nkv, maps, hd, vd, \
                       v_off, v_is_k, write_kv, status))))
        if (widest <= 128) { if (hpw == 1) FB_QKR_HEADS(1, 1); else FB_QKR_HEADS(1, 4); }
        else if (widest <= 256) { if (hpw == 1) FB_QKR_HEADS(2, 1); else FB_QKR_HEADS(2, 4); }
        else { if (hpw == 1) FB_QKR_HEADS(4, 1); else FB_QKR_HEADS(4, 4); }
#undef FB_QKR_HEADS
        return fb_check_launch("qk_norm_rope_kv_write");
    }
    const size_t smem = ((size_t)(nh + nkv) * hd + nh + nkv) * sizeof(float);
    FB_REQUIRE(smem <= 200 * 1024, "qk_norm_rope_kv_write: a row of q and k (%zu bytes) does not fit shared memory", smem);
    FB_DISPATCH_DTYPE(w_dtype, TW, FB_DISPATCH_DTYPE(out_dtype, T, {
        auto kernel = qk_norm_rope_kv_write_kernel<TW, T>;
        if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        const int cols = (nh + 2 * nkv) * (hd > vd ? hd : vd);
        fb_launch(kernel, dim3(n), dim3(n > 128 ? 256 : cols >= 4096 ? 1024 : cols >= 1024 ? 512 : 256), smem, stream, proj, (long)proj_stride, n_partials, (long)partial_stride,
                  (const TW*)bias, (const TW*)q_weight, (const TW*)k_weight, scope, eps, weight_offset, cos_t, sin_t, half, (T*)q_out,
                  (long)q_out_stride, positions, row_seq, block_table, table_stride, table_base, table_head, (T*)k_pool,
                  (T*)v_pool, page_size, n_pages, nh, nkv, maps, hd, vd, v_off, write_kv, status);
    }));
    return fb_check_launch("qk_norm_rope_kv_write");
}
