// What a token's id gives to the stream besides its embedding row.
//
//   embedding_pairs   x[t] = E[id[t]] * scale + P[row], row = (a * id of the token before + b * id[t]) mod buckets, and
//                     the row behind the buckets for a request's first token.  The token before the step's first one
//                     lies in the request's state slot (its id + 1; 0: there is none); the CTA of an entry's first row
//                     reads it and leaves the entry's last id there for the next step.
//   token_gate        g[t] = gelu(z[t]) * T[id[t]][offset ..]: the gate of a layer's token input, z being a product that
//                     arrives as float32 split-K shares; columns behind `dim` (padding of the product) become zero.
#include "rows.cuh"

template <typename TT, int VEC>
__global__ void __launch_bounds__(256)
embedding_pairs_kernel(const TT* __restrict__ table, const TT* __restrict__ pairs, const int* __restrict__ ids,
                       const int* __restrict__ row_seq, const int* __restrict__ seq_q_start,
                       const int* __restrict__ seq_q_len, const int* __restrict__ seq_slot, int* __restrict__ state,
                       long state_stride, long long mul_prev, long long mul_cur, int buckets, float* __restrict__ x,
                       int H, int V, float scale, int* status) {
    fb_pdl_launch_dependents();
    fb_pdl_wait();
    __shared__ int before;                             // the id of the token before this row's + 1; 0: there is none
    const int t = blockIdx.x;
    int id = ids[t];
    if (threadIdx.x == 0) {
        const int seq = row_seq[t], start = seq_q_start[seq];
        int b;
        if (t > start) {
            b = ids[t - 1] + 1;
        } else {
            int* kept = state + (size_t)seq_slot[seq] * state_stride;
            b = *kept;
            *kept = ids[start + seq_q_len[seq] - 1] + 1;
        }
        if (id < 0 || id >= V || b < 0 || b > V) {
            atomicOr(status, FB_STATUS_BAD_TOKEN);
            b = 0;
        }
        before = b;
    }
    __syncthreads();
    if (id < 0 || id >= V) id = 0;
    const int b = before;
    const long row = b > 0 ? (long)((mul_prev * (b - 1) + mul_cur * id) % buckets) : buckets;
    const TT* e = table + (size_t)id * H;
    const TT* p = pairs + (size_t)row * H;
    float* dst = x + (size_t)t * H;
    for (int c = threadIdx.x * VEC; c < H; c += blockDim.x * VEC) {
        if constexpr (VEC == 4) {
            const float4 u = Vec4<TT>::load(e + c), v = Vec4<TT>::load(p + c);
            Vec4<float>::store(dst + c, make_float4(fmaf(u.x, scale, v.x), fmaf(u.y, scale, v.y), fmaf(u.z, scale, v.z),
                                                    fmaf(u.w, scale, v.w)));
        } else {
            dst[c] = fmaf(fb_to_float(e[c]), scale, fb_to_float(p[c]));
        }
    }
}

// table [V, H] and pairs [buckets + 1, H] share a dtype; 0 <= mul_prev, mul_cur < buckets (residues serve as well as
// the numbers themselves, and keep the sum far from the end of 64 bits).  state: int32, one per slot `state_stride` apart.
FB_API int fb_embedding_pairs(const void* table, const void* pairs, int table_dtype, const int* ids, const int* row_seq,
                              const int* seq_q_start, const int* seq_q_len, const int* seq_slot, int* state,
                              long long state_stride, long long mul_prev, long long mul_cur, int buckets, float* x,
                              int n, int H, int V, float scale, int* status, cudaStream_t stream) {
    FB_REQUIRE(n >= 0 && H > 0 && V > 0 && buckets > 0, "embedding_pairs: bad sizes n=%d H=%d V=%d buckets=%d", n, H, V, buckets);
    FB_REQUIRE(mul_prev >= 0 && mul_prev < buckets && mul_cur >= 0 && mul_cur < buckets,
               "embedding_pairs: the factors are residues of the buckets");
    FB_REQUIRE(pairs && state && row_seq && seq_q_start && seq_q_len && seq_slot, "embedding_pairs: arguments missing");
    if (n == 0) return 0;
    const bool vec = H % 4 == 0 && (uintptr_t)table % 16 == 0 && (uintptr_t)pairs % 16 == 0 && (uintptr_t)x % 16 == 0;
    const int threads = H >= 1024 ? 256 : 128;
    FB_DISPATCH_DTYPE(table_dtype, TT, {
        if (vec)
            fb_launch((embedding_pairs_kernel<TT, 4>), n, threads, 0, stream, (const TT*)table, (const TT*)pairs, ids, row_seq,
                      seq_q_start, seq_q_len, seq_slot, state, (long)state_stride, mul_prev, mul_cur, buckets, x, H, V,
                      scale, status);
        else
            fb_launch((embedding_pairs_kernel<TT, 1>), n, threads, 0, stream, (const TT*)table, (const TT*)pairs, ids, row_seq,
                      seq_q_start, seq_q_len, seq_slot, state, (long)state_stride, mul_prev, mul_cur, buckets, x, H, V,
                      scale, status);
    });
    return fb_check_launch("embedding_pairs");
}

template <typename TT, typename TO, int VEC>
__global__ void __launch_bounds__(256)
token_gate_kernel(const float* __restrict__ z, long z_stride, int n_partials, long partial_stride,
                  const TT* __restrict__ table, long table_stride, int offset, const int* __restrict__ ids, int V,
                  TO* __restrict__ out, int n, int dim, int cols, int* status) {
    fb_pdl_launch_dependents();
    const int per = cols / VEC;
    const size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    const int t = (int)(idx / per), c = (int)(idx - (size_t)t * per) * VEC;
    fb_pdl_wait();
    if (t >= n) return;
    int id = ids[t];
    if (id < 0 || id >= V) {
        atomicOr(status, FB_STATUS_BAD_TOKEN);
        id = 0;
    }
    const TT* e = table + (size_t)id * table_stride + offset + c;
    const float* zr = z + (size_t)t * z_stride + c;
    TO* o = out + (size_t)t * cols + c;
    if constexpr (VEC == 4) {                          // dim is a multiple of 4: a thread's columns are all in or all out
        float4 g = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < dim) {
            const float4 u = Vec4<TT>::load(e);
            g = slab_sum4(zr, n_partials, partial_stride);
            g.x = fb_gelu_tanh(g.x) * u.x; g.y = fb_gelu_tanh(g.y) * u.y;
            g.z = fb_gelu_tanh(g.z) * u.z; g.w = fb_gelu_tanh(g.w) * u.w;
        }
        Vec4<TO>::store(o, g);
    } else {
        o[0] = fb_from_float<TO>(c < dim ? fb_gelu_tanh(fb_slab_sum(zr, 0, n_partials, partial_stride)) * fb_to_float(e[0]) : 0.0f);
    }
}

// z: float32 [n, >= dim] (possibly shares); table [V, table_stride], of which a layer reads `dim` columns from `offset`
// on; out [n, cols] contiguous, cols >= dim.
FB_API int fb_token_gate(const float* z, long long z_stride, int n_partials, long long partial_stride, const void* table,
                         int table_dtype, long long table_stride, int offset, const int* ids, int V, void* out,
                         int out_dtype, int n, int dim, int cols, int* status, cudaStream_t stream) {
    FB_REQUIRE(n >= 0 && dim > 0 && cols >= dim && z_stride >= dim && V > 0, "token_gate: bad sizes n=%d dim=%d", n, dim);
    FB_REQUIRE(offset >= 0 && table_stride >= (long long)offset + dim, "token_gate: the table's rows are too short");
    if (n == 0) return 0;
    if (n_partials < 1) n_partials = 1;
    const bool vec = dim % 4 == 0 && cols % 4 == 0 && z_stride % 4 == 0 && partial_stride % 4 == 0 && offset % 4 == 0 &&
                     table_stride % 4 == 0 && (uintptr_t)z % 16 == 0 && (uintptr_t)table % 16 == 0 && (uintptr_t)out % 16 == 0;
    const size_t total = (size_t)n * (vec ? cols / 4 : cols);
    FB_DISPATCH_DTYPE(table_dtype, TT, FB_DISPATCH_DTYPE(out_dtype, TO, {
        if (vec)
            fb_launch((token_gate_kernel<TT, TO, 4>), (unsigned)((total + 255) / 256), 256, 0, stream, z, (long)z_stride,
                      n_partials, (long)partial_stride, (const TT*)table, (long)table_stride, offset, ids, V, (TO*)out, n,
                      dim, cols, status);
        else
            fb_launch((token_gate_kernel<TT, TO, 1>), (unsigned)((total + 255) / 256), 256, 0, stream, z, (long)z_stride,
                      n_partials, (long)partial_stride, (const TT*)table, (long)table_stride, offset, ids, V, (TO*)out, n,
                      dim, cols, status);
    }));
    return fb_check_launch("token_gate");
}
