// Layer norm with a weight and no bias (before a sublayer), fused with the pending residual additions.
//
//   v = x[row] + delta[row] + more_rows[row] + more_vec        (each addend optional)
//   h = (v - mean(v)) / sqrt(mean((v - mean(v))^2) + eps) * w
//
// rows == nullptr: every row t; x[t] is replaced by v (the residual stream moves on).
// rows != nullptr: for i < n_rows the row rows[i] is read and h[i] written; x stays.
//
// delta is a tensor of either element type, or (delta_parts > 1) that many float32
// slices part_stride elements apart (a matrix product cut along K), added in the order
// of the slices.  more_rows is float32 [T, d] (a second stream added row by row, e.g.
// the embedding's output at the start of a repeated pass), more_vec one vector [d]
// added to every row.
//
// Everything is float32 with one rounding at the store.  Mean and variance are taken
// in two passes over the row held in shared memory; the order of both sums depends on
// d alone (one block of LN_THREADS threads a row), so a row's result does not depend
// on the batch it is in.
//
// mls_add_post_layernorm is the other arrangement, a norm behind a sublayer:
//
//   y = the sublayer's result at row t (a tensor, or the sum of K-parts) + y_bias      (optional)
//   y = (y - mean(y)) / sqrt(mean((y - mean(y))^2) + eps) * w1 + b1
//   v = x[t] + y                                    (x may be absent: v = y)
//   h = v, or a second such norm of v with w2, b2   (h may be absent)
//
// without `rows` for every row t, x[t] = v; with rows only those are read and x stays.  The row
// stays in registers; which thread holds which entries depends on the row's width alone.
//
// mls_residual_add only settles more_rows / more_vec into x, for a norm of another kind.
#include "common.cuh"
#include "row_pack.cuh"

namespace {
constexpr int LN_THREADS = 256;

__global__ void __launch_bounds__(LN_THREADS)
add_layernorm_kernel(float* __restrict__ x, const void* __restrict__ delta, int delta_dtype,
                     int delta_parts, size_t part_stride, const float* __restrict__ more_rows,
                     const void* __restrict__ more_vec, int vec_dtype,
                     const void* __restrict__ w, int w_dtype, float eps, void* __restrict__ h,
                     int h_dtype, int n_rows, int d, const int* __restrict__ rows) {
    chain_release();
    chain_wait();
    extern __shared__ float row_s[];
    __shared__ float scratch[33];
    for (int out_row = blockIdx.x; out_row < n_rows; out_row += gridDim.x) {
        const size_t src = (size_t)(rows ? rows[out_row] : out_row) * d;
        float s = 0.f;
        for (int c = threadIdx.x; c < d; c += LN_THREADS) {
            float v = x[src + c];
            if (delta) {
                float a = load_as_float(delta, src + c, delta_parts > 1 ? MLS_F32 : delta_dtype);
                for (int k = 1; k < delta_parts; ++k)
                    a += ((const float*)delta)[src + c + (size_t)k * part_stride];
                v += a;
            }
            if (more_rows) v += more_rows[src + c];
            if (more_vec) v += load_as_float(more_vec, c, vec_dtype);
            row_s[c] = v;
            if (!rows) x[src + c] = v;
            s += v;
        }
        const float mean = block_sum(s, scratch) / (float)d;
        float q = 0.f;
        for (int c = threadIdx.x; c < d; c += LN_THREADS) {
            const float u = row_s[c] - mean;
            q = fmaf(u, u, q);
        }
        const float var = block_sum(q, scratch) / (float)d;
        const float inv = 1.0f / sqrtf(var + eps);
        for (int c = threadIdx.x; c < d; c += LN_THREADS)
            store_from_float(h, (size_t)out_row * d + c, h_dtype,
                             (row_s[c] - mean) * inv * load_as_float(w, c, w_dtype));
        __syncthreads();                         // row_s is filled again for the next row
    }
}

__global__ void residual_add_kernel(float* __restrict__ x, const float* __restrict__ more_rows,
                                    const void* __restrict__ more_vec, int vec_dtype,
                                    size_t n, int d) {
    chain_release();
    chain_wait();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n;
         i += (size_t)gridDim.x * blockDim.x) {
        float v = x[i];
        if (more_rows) v += more_rows[i];
        if (more_vec) v += load_as_float(more_vec, i % d, vec_dtype);
        x[i] = v;
    }
}

// x += delta (a tensor, the parts of a product cut along K, or nothing); then
// out[t] = [x[t] | other[t]] in the activation type: the input of a projection that reads
// the stream beside a second stream.
__global__ void settle_concat_kernel(float* __restrict__ x, const void* __restrict__ delta,
                                     int delta_dtype, int n_parts, size_t part_stride,
                                     const float* __restrict__ other, void* __restrict__ out,
                                     int out_dtype, size_t n, int d) {
    chain_release();
    chain_wait();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n;
         i += (size_t)gridDim.x * blockDim.x) {
        float v = x[i];
        if (delta) {
            float add = 0.f;
            for (int k = 0; k < n_parts; ++k)
                add += load_as_float(delta, i + (size_t)k * part_stride, delta_dtype);
            v += add;
            x[i] = v;
        }
        const size_t t = i / d, c = i - t * d;
        store_from_float(out, t * 2 * d + c, out_dtype, v);
        store_from_float(out, t * 2 * d + d + c, out_dtype, other[i]);
    }
}

struct PostNormArgs {
    float* x;
    const void* y;                     // [parts][T, d] or nullptr: no sublayer's result
    int y_dtype, y_parts;
    long long y_stride;
    const float *y_bias, *w1, *b1, *w2, *b2;      // [d]; y_bias and (w2, b2) may be absent
    float eps;
    void* h;
    int h_dtype;
    float* y_out;
    const int* rows;
    int d;
};

// Sum over the block with one barrier; `scratch` belongs to this sum alone.  Every thread adds
// the warps' sums in their order.
__device__ __forceinline__ float row_sum(float v, float* scratch /* >= 32 floats */) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = v;
    __syncthreads();
    float s = 0.f;
    const int n = (int)(blockDim.x >> 5);
    for (int i = 0; i < n; ++i) s += scratch[i];
    return s;
}

// Layer norm of a row held as packs; the vectors are held already (HELD) or read where needed.
template <int N, int VEC, bool HELD>
__device__ __forceinline__ void norm_packs(Pack<N> (&v)[VEC], const Pack<N> (&w)[HELD ? VEC : 1],
                                           const Pack<N> (&b)[HELD ? VEC : 1],
                                           const float* __restrict__ pw,
                                           const float* __restrict__ pb, int d, float eps,
                                           float* scratch /* >= 64 floats */) {
    float s = 0.f, q = 0.f;
#pragma unroll
    for (int k = 0; k < VEC; ++k)
        if (((int)threadIdx.x + k * (int)blockDim.x) * N < d)
#pragma unroll
            for (int e = 0; e < N; ++e) s += v[k].v[e];
    const float mean = row_sum(s, scratch) / (float)d;
#pragma unroll
    for (int k = 0; k < VEC; ++k)
        if (((int)threadIdx.x + k * (int)blockDim.x) * N < d)
#pragma unroll
            for (int e = 0; e < N; ++e) {
                v[k].v[e] -= mean;
                q = fmaf(v[k].v[e], v[k].v[e], q);
            }
    const float inv = 1.0f / sqrtf(row_sum(q, scratch + 32) / (float)d + eps);
#pragma unroll
    for (int k = 0; k < VEC; ++k) {
        const int c = ((int)threadIdx.x + k * (int)blockDim.x) * N;
        if (c < d) {
            const Pack<N> wk = HELD ? w[HELD ? k : 0] : load_pack<N>(pw, c, MLS_F32);
            const Pack<N> bk = HELD ? b[HELD ? k : 0] : load_pack<N>(pb, c, MLS_F32);
#pragma unroll
            for (int e = 0; e < N; ++e) v[k].v[e] = fmaf(v[k].v[e] * inv, wk.v[e], bk.v[e]);
        }
    }
}

// N: entries a thread takes at a time (4 where every row starts at a 16-byte place), VEC: such
// groups a thread holds, threads * N * VEC >= d.  FEW: few rows; K-parts are possible and the
// norm's vectors are read ahead of the wait on the kernel before.
template <int N, int VEC, int MAX_THREADS, bool FEW>
__global__ void __launch_bounds__(MAX_THREADS, (FEW || MAX_THREADS > 256) ? 1 : VEC <= 2 ? 4 : VEC <= 4 ? 3 : 1)
add_post_layernorm_kernel(const PostNormArgs a) {
    chain_release();
    __shared__ float scratch[4][32];
    const int i = blockIdx.x, d = a.d;
    const int t = a.rows ? a.rows[i] : i;
    const size_t at = (size_t)t * d;
    constexpr bool HELD = FEW && MAX_THREADS <= 256;
    Pack<N> y[VEC], x[VEC], w[HELD ? VEC : 1], b[HELD ? VEC : 1], none[1];
    if constexpr (HELD) {
        if (a.y) {
#pragma unroll
            for (int k = 0; k < VEC; ++k) {
                const int c = ((int)threadIdx.x + k * (int)blockDim.x) * N;
                if (c < d) {
                    w[k] = load_pack<N>(a.w1, c, MLS_F32);
                    b[k] = load_pack<N>(a.b1, c, MLS_F32);
                }
            }
        }
    }
    chain_wait();
#pragma unroll
    for (int k = 0; k < VEC; ++k) {
        const int c = ((int)threadIdx.x + k * (int)blockDim.x) * N;
        if (c < d) {
            if (a.y) {
                y[k] = load_parts<N>(a.y, at + c, a.y_dtype, FEW ? a.y_parts : 1, (size_t)a.y_stride);
                if (a.y_bias) {
                    const Pack<N> bias = load_pack<N>(a.y_bias, c, MLS_F32);
#pragma unroll
                    for (int e = 0; e < N; ++e) y[k].v[e] += bias.v[e];
                }
            }
            if (a.x) x[k] = load_pack<N>(a.x, at + c, MLS_F32);
        }
    }
    if (a.y) norm_packs<N, VEC, HELD>(y, w, b, a.w1, a.b1, d, a.eps, scratch[0]);
#pragma unroll
    for (int k = 0; k < VEC; ++k) {
        const int c = ((int)threadIdx.x + k * (int)blockDim.x) * N;
        if (c < d) {
            if (a.y_out) store_pack<N>(a.y_out, (size_t)i * d + c, MLS_F32, y[k]);
            if (!a.x) {
                x[k] = y[k];
            } else if (a.y) {
#pragma unroll
                for (int e = 0; e < N; ++e) x[k].v[e] += y[k].v[e];
                if (!a.rows) store_pack<N>(a.x, at + c, MLS_F32, x[k]);
            }
        }
    }
    if (!a.h) return;
    if (a.w2) norm_packs<N, VEC, false>(x, none, none, a.w2, a.b2, d, a.eps, scratch[2]);
#pragma unroll
    for (int k = 0; k < VEC; ++k) {
        const int c = ((int)threadIdx.x + k * (int)blockDim.x) * N;
        if (c < d) store_pack<N>(a.h, (size_t)i * d + c, a.h_dtype, x[k]);
    }
}
}  // namespace

MLS_API int mls_add_post_layernorm(float* x, const void* y, int y_dtype, int y_parts,
                                   long long y_stride, const float* y_bias, const float* w1,
                                   const float* b1, const float* w2, const float* b2, float eps,
                                   void* h, int h_dtype, float* y_out, const int* rows, int n_out,
                                   int d, cudaStream_t stream) {
    if (n_out <= 0 || d <= 0) return 0;
    if ((y && (!w1 || !b1)) || (!x && !y) || (w2 && !b2) || y_parts < 1 || (y_out && !y) ||
        (y_parts > 1 && y_dtype != MLS_F32))
        return MLS_ERR_UNSUPPORTED;
    PostNormArgs a;
    a.x = x; a.y = y; a.y_dtype = y_dtype; a.y_parts = y_parts; a.y_stride = y_stride;
    a.y_bias = y_bias; a.w1 = w1; a.b1 = b1; a.w2 = w2; a.b2 = b2; a.eps = eps; a.h = h;
    a.h_dtype = h_dtype; a.y_out = y_out; a.rows = rows; a.d = d;
    // four entries a thread where every row and vector starts at a 16-byte place (buffers do:
    // this depends on the model's sizes)
    uintptr_t bits = 0;
    for (const void* p : {(const void*)x, y, (const void*)y_bias, (const void*)w1, (const void*)b1,
                          (const void*)w2, (const void*)b2, (const void*)h, (const void*)y_out})
        bits |= reinterpret_cast<uintptr_t>(p);
    const bool by4 = d % 4 == 0 && bits % 16 == 0 && (y_parts == 1 || y_stride % 4 == 0);
    const int groups = by4 ? d / 4 : d;
    // few groups: a group a thread, up to 256 threads; then up to four groups a thread; then
    // more threads
    int threads = 32;
    while (threads < 256 && threads < groups) threads <<= 1;
    while (threads < 1024 && threads * 4 < groups) threads <<= 1;
    const int vec = (groups + threads - 1) / threads;
    const bool few = y_parts > 1 || n_out <= 2 * sm_count();
#define PN_RUN(N, V, M, F) \
    MLS_LAUNCH((add_post_layernorm_kernel<N, V, M, F>), dim3(n_out), dim3(threads), 0, stream, a)
#define PN_GO(N, V)                                  \
    do {                                             \
        if (threads > 256) PN_RUN(N, V, 1024, true); \
        else if (few) PN_RUN(N, V, 256, true);       \
        else PN_RUN(N, V, 256, false);               \
    } while (0)
    if (by4) {
        if (vec <= 1) PN_GO(4, 1);
        else if (vec <= 2) PN_GO(4, 2);
        else if (vec <= 4) PN_GO(4, 4);
        else return MLS_ERR_UNSUPPORTED;
    } else {
        if (vec <= 1) PN_GO(1, 1);
        else if (vec <= 4) PN_GO(1, 4);
        else if (vec <= 16) PN_GO(1, 16);
        else return MLS_ERR_UNSUPPORTED;
    }
#undef PN_GO
#undef PN_RUN
    return launch_status();
}

MLS_API int mls_settle_concat(float* x, const void* delta, int delta_dtype, int delta_parts,
                              long long part_stride, const float* other, void* out,
                              int out_dtype, int n_rows, int d, cudaStream_t stream) {
    if (n_rows <= 0 || d <= 0) return 0;
    const size_t n = (size_t)n_rows * d;
    const int blocks = (int)((n + 255) / 256 < (size_t)(8 * sm_count()) ? (n + 255) / 256
                                                                       : 8 * sm_count());
    MLS_LAUNCH((settle_concat_kernel), dim3(blocks), dim3(256), 0, stream, x, delta, delta_dtype,
               delta_parts < 1 ? 1 : delta_parts, (size_t)part_stride, other, out, out_dtype, n,
               d);
    return launch_status();
}

MLS_API int mls_add_layernorm(float* x, const void* delta, int delta_dtype, int delta_parts,
                              long long part_stride, const float* more_rows, const void* more_vec,
                              int vec_dtype, const void* w, int w_dtype, float eps, void* h,
                              int h_dtype, int n_rows, int d, const int* rows,
                              cudaStream_t stream) {
    if (n_rows <= 0 || d <= 0) return 0;
    const size_t smem = (size_t)d * sizeof(float);
    if (smem > 200 * 1024) return MLS_ERR_UNSUPPORTED;
    if (smem > 48 * 1024) {
        const int rc = (int)cudaFuncSetAttribute(add_layernorm_kernel,
                                                 cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                 (int)smem);
        if (rc) return rc;
    }
    const int blocks = n_rows < 8 * sm_count() ? n_rows : 8 * sm_count();
    MLS_LAUNCH((add_layernorm_kernel), dim3(blocks), dim3(LN_THREADS), smem, stream, x, delta,
               delta_dtype, delta_parts < 1 ? 1 : delta_parts, (size_t)part_stride, more_rows,
               more_vec, vec_dtype, w, w_dtype, eps, h, h_dtype, n_rows, d, rows);
    return launch_status();
}

MLS_API int mls_residual_add(float* x, const float* more_rows, const void* more_vec,
                             int vec_dtype, int n_rows, int d, cudaStream_t stream) {
    if (n_rows <= 0 || d <= 0 || (!more_rows && !more_vec)) return 0;
    const size_t n = (size_t)n_rows * d;
    const int blocks = (int)((n + 255) / 256 < (size_t)(8 * sm_count()) ? (n + 255) / 256
                                                                       : 8 * sm_count());
    MLS_LAUNCH((residual_add_kernel), dim3(blocks), dim3(256), 0, stream, x, more_rows, more_vec,
               vec_dtype, n, d);
    return launch_status();
}
