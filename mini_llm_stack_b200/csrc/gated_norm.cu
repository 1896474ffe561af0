// What stands between a sublayer and the next one when the sublayer's result is gated and normed
// before it joins the residual stream: one kernel, one pass over the row.
//
// mls_add_gated_norm, for every output row i (source row t = rows ? rows[i] : i):
//   y = the sublayer's result at row t (a tensor, or the sum of a product's K-parts)
//   if gate:  y *= sigmoid(z + gate_bias), z the gate's pre-activation (columns of float32 or
//             bfloat16 rows, or K-parts; the bias is optional)
//   y = y / sqrt(mean(y^2) + eps) * post_w
//   v = x[t] + y;  without `rows`, x[t] = v                    (x may be absent: v = y)
//   h[i] = v / sqrt(mean(v^2) + eps) * pre_w                   (h may be absent)
//   y_out[i] = y                                               (y_out may be absent)
// A norm's weight is a vector, or one number for all coordinates (its step is then 0).
// Everything is float32 inside, one rounding at the store of h.  One block a row; which thread
// holds which entries, and with it the order of the sums, depends on the row's width alone.
#include "common.cuh"
#include "row_pack.cuh"

namespace {
struct GatedNormArgs {
    float* x;
    const void* y;                     // [parts][T, d]
    int y_dtype, y_parts;
    long long y_stride;
    const void* z;                     // [parts][T, z_row], or nullptr: no gate
    int z_dtype, z_parts, z_row, z_col;
    long long z_stride;
    const float* z_bias;               // [d] or nullptr
    const float* post_w;               // [d], or one number
    const float* pre_w;
    int post_step, pre_step;           // 1: a vector, 0: one number
    float eps;
    void* h;
    int h_dtype;
    float* y_out;
    const int* rows;
    int n_out, d;
};

__device__ __forceinline__ float sigmoid1(float z) { return 1.0f / (1.0f + expf(-z)); }

template <int N>
__device__ __forceinline__ Pack<N> weight_pack(const float* w, int step, int c) {
    if (step) return load_pack<N>(w, c, MLS_F32);
    Pack<N> r;
#pragma unroll
    for (int e = 0; e < N; ++e) r.v[e] = w[0];
    return r;
}
// N: entries a thread takes at a time (4: every row starts at a 16-byte place; else 1).
// VEC: such groups a thread keeps in registers, threads * N * VEC >= d.  PARTS: the result or
// the gate may come as K-parts (few rows); without, the kernel has registers for more blocks an
// SM, whose rows' loads and block sums then overlap.
constexpr int blocks_an_sm(int vec, int max_threads, bool parts) {
    return parts || max_threads > 256 ? 1 : vec <= 1 ? 6 : vec <= 2 ? 5 : vec <= 4 ? 3 : 1;
}
template <int N, int VEC, int MAX_THREADS, bool PARTS>
__global__ void __launch_bounds__(MAX_THREADS, blocks_an_sm(VEC, MAX_THREADS, PARTS))
add_gated_norm_kernel(const GatedNormArgs a) {
    chain_release();
    __shared__ float scratch[33];
    const int groups = a.d / N, i = blockIdx.x;
    const int t = a.rows ? a.rows[i] : i;
    chain_wait();
    const size_t at = (size_t)t * a.d;
    Pack<N> y[VEC], x[VEC];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < VEC; ++k) {
        const int c = ((int)threadIdx.x + k * (int)blockDim.x) * N;
        if (c < groups * N) {
            y[k] = load_parts<N>(a.y, at + c, a.y_dtype, PARTS ? a.y_parts : 1, (size_t)a.y_stride);
            if (a.x) x[k] = load_pack<N>(a.x, at + c, MLS_F32);
            if (a.z) {
                Pack<N> z = load_parts<N>(a.z, (size_t)t * a.z_row + a.z_col + c, a.z_dtype,
                                          PARTS ? a.z_parts : 1, (size_t)a.z_stride);
                if (a.z_bias) {
                    const Pack<N> b = load_pack<N>(a.z_bias, c, MLS_F32);
#pragma unroll
                    for (int e = 0; e < N; ++e) z.v[e] += b.v[e];
                }
#pragma unroll
                for (int e = 0; e < N; ++e) y[k].v[e] *= sigmoid1(z.v[e]);
            }
#pragma unroll
            for (int e = 0; e < N; ++e) ss = fmaf(y[k].v[e], y[k].v[e], ss);
        }
    }
    const float inv_y = 1.0f / sqrtf(block_sum(ss, scratch) / (float)a.d + a.eps);
    ss = 0.f;
#pragma unroll
    for (int k = 0; k < VEC; ++k) {
        const int c = ((int)threadIdx.x + k * (int)blockDim.x) * N;
        if (c < groups * N) {
            const Pack<N> w = weight_pack<N>(a.post_w, a.post_step, c);
#pragma unroll
            for (int e = 0; e < N; ++e) y[k].v[e] = y[k].v[e] * inv_y * w.v[e];
            if (a.y_out) store_pack<N>(a.y_out, (size_t)i * a.d + c, MLS_F32, y[k]);
            if (a.x) {
#pragma unroll
                for (int e = 0; e < N; ++e) x[k].v[e] += y[k].v[e];
                if (!a.rows) store_pack<N>(a.x, at + c, MLS_F32, x[k]);
            } else {
                x[k] = y[k];
            }
#pragma unroll
            for (int e = 0; e < N; ++e) ss = fmaf(x[k].v[e], x[k].v[e], ss);
        }
    }
    if (!a.h) return;
    const float inv_x = 1.0f / sqrtf(block_sum(ss, scratch) / (float)a.d + a.eps);
#pragma unroll
    for (int k = 0; k < VEC; ++k) {
        const int c = ((int)threadIdx.x + k * (int)blockDim.x) * N;
        if (c < groups * N) {
            const Pack<N> w = weight_pack<N>(a.pre_w, a.pre_step, c);
#pragma unroll
            for (int e = 0; e < N; ++e) x[k].v[e] = x[k].v[e] * inv_x * w.v[e];
            store_pack<N>(a.h, (size_t)i * a.d + c, a.h_dtype, x[k]);
        }
    }
}
}  // namespace

MLS_API int mls_add_gated_norm(float* x, const void* y, int y_dtype, int y_parts, long long y_stride,
                               const void* z, int z_dtype, int z_parts, long long z_stride, int z_row,
                               int z_col, const float* z_bias, const float* post_w, int post_step,
                               const float* pre_w, int pre_step, float eps, void* h, int h_dtype,
                               float* y_out, const int* rows, int n_out, int d,
                               cudaStream_t stream) {
    if (n_out <= 0 || d <= 0) return 0;
    if (!y || !post_w || (h && !pre_w) || y_parts < 1 || (z && z_parts < 1) ||
        (y_parts > 1 && y_dtype != MLS_F32) || (z && z_parts > 1 && z_dtype != MLS_F32))
        return MLS_ERR_UNSUPPORTED;
    GatedNormArgs a;
    a.x = x; a.y = y; a.y_dtype = y_dtype; a.y_parts = y_parts; a.y_stride = y_stride;
    a.z = z; a.z_dtype = z_dtype; a.z_parts = z_parts; a.z_stride = z_stride; a.z_row = z_row;
    a.z_col = z_col; a.z_bias = z_bias; a.post_w = post_w; a.post_step = post_step; a.pre_w = pre_w;
    a.pre_step = pre_step; a.eps = eps; a.h = h; a.h_dtype = h_dtype; a.y_out = y_out; a.rows = rows;
    a.n_out = n_out; a.d = d;
    // four entries a thread where every row and vector starts at a 16-byte place (buffers do:
    // this depends on the model's sizes)
    uintptr_t bits = 0;
    for (const void* p : {(const void*)x, y, z, (const void*)z_bias, (const void*)h, (const void*)y_out,
                          post_step ? (const void*)post_w : nullptr,
                          pre_step ? (const void*)pre_w : nullptr})
        bits |= reinterpret_cast<uintptr_t>(p);
    const bool by4 = d % 4 == 0 && bits % 16 == 0 && (y_parts == 1 || y_stride % 4 == 0) &&
                     (!z || (z_row % 4 == 0 && z_col % 4 == 0 && (z_parts == 1 || z_stride % 4 == 0)));
    const int groups = by4 ? d / 4 : d;
    // few groups: a group a thread, up to 256 threads; then up to four groups a thread; then
    // more threads
    int threads = 32;
    while (threads < 256 && threads < groups) threads <<= 1;
    while (threads < 1024 && threads * 4 < groups) threads <<= 1;
    const int vec = (groups + threads - 1) / threads;
    if (vec > 16) return MLS_ERR_UNSUPPORTED;
    const bool parts = y_parts > 1 || (z && z_parts > 1);
#define GN_RUN(N, V, M, P) \
    MLS_LAUNCH((add_gated_norm_kernel<N, V, M, P>), dim3(n_out), dim3(threads), 0, stream, a)
#define GN_GO(N, V)                                \
    do {                                           \
        if (threads > 256) GN_RUN(N, V, 1024, true); \
        else if (parts) GN_RUN(N, V, 256, true);   \
        else GN_RUN(N, V, 256, false);             \
    } while (0)
    if (by4) {
        if (vec <= 1) GN_GO(4, 1);
        else if (vec <= 2) GN_GO(4, 2);
        else if (vec <= 4) GN_GO(4, 4);
        else if (vec <= 8) GN_GO(4, 8);
        else return MLS_ERR_UNSUPPORTED;
    } else {
        if (vec <= 1) GN_GO(1, 1);
        else if (vec <= 4) GN_GO(1, 4);
        else GN_GO(1, 16);
    }
#undef GN_GO
#undef GN_RUN
    return launch_status();
}
