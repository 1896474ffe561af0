// Causal grouped-query attention over the paged cache on CUDA cores, for any
// mix of prompt portions and single decoded tokens.  It serves the float32 path
// (everything in 32-bit) and checks the tensor-core kernels of the bfloat16 path.
//
// Reference math (train/model.py:55-70): S = (q . k) * scale in float32; key j is
// hidden from the query at absolute position p iff j > p (the bottom-right
// aligned causal mask with p = i + Sk - Sq); P = softmax(S); O = P . V in
// float32, rounded once.  q head h reads kv head h / G.  With a window w, keys
// j <= p - w are hidden too.  With a cap c > 0 the score becomes c * tanh(S / c) before
// the softmax.  With sinks (one learned number per q head) the softmax's denominator also
// holds exp(sink_h): a term without key or value, not scaled and not capped.  With slopes
// (one number per q head) the score loses slope_h * (p - j), the distance to the key, before
// the cap.  With keep_first > 0 a window does not hide the sequence's first keep_first keys.
// With chunks of c tokens (and no window) the query at position p sees its own chunk, keys
// floor(p / c) c .. p.
// A row of `out` may be wider than the heads (out_stride elements a token).  The paged walk follows the reference's decode
// kernel (kernels/paged_attention.py:34-88): page = table[r, j / block],
// offset = j % block, online softmax over chunks of keys.
//
// One warp per (token, q head).  Keys are taken 32 at a time from an absolute
// multiple of 32, so the order of every sum depends only on the token's own
// position and window: the result is bit-for-bit the same however the tokens
// were cut into steps and whatever else is in the batch.
#include "common.cuh"

namespace {
constexpr int WARPS = 4;
constexpr int MOST_HD = 1024;         // heads of up to 512 entries take a smaller instantiation

// q . k over one key row, accumulated in the order i = 0 .. hd-1.
__device__ __forceinline__ float dot_row(const float* q, const float* k, int hd) {
    float dot = 0.f;
    if ((hd & 3) == 0) {
        for (int i = 0; i < hd; i += 4) {
            const float4 v = *reinterpret_cast<const float4*>(k + i);
            dot = fmaf(q[i], v.x, dot);
            dot = fmaf(q[i + 1], v.y, dot);
            dot = fmaf(q[i + 2], v.z, dot);
            dot = fmaf(q[i + 3], v.w, dot);
        }
    } else {
        for (int i = 0; i < hd; ++i) dot = fmaf(q[i], k[i], dot);
    }
    return dot;
}
__device__ __forceinline__ float dot_row(const float* q, const __nv_bfloat16* k, int hd) {
    float dot = 0.f;
    if ((hd & 7) == 0) {
        for (int i = 0; i < hd; i += 8) {
            const uint4 raw = *reinterpret_cast<const uint4*>(k + i);
            const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float2 f = __bfloat1622float2(h2[e]);
                dot = fmaf(q[i + 2 * e], f.x, dot);
                dot = fmaf(q[i + 2 * e + 1], f.y, dot);
            }
        }
    } else {
        for (int i = 0; i < hd; ++i) dot = fmaf(q[i], __bfloat162float(k[i]), dot);
    }
    return dot;
}

template <typename T, int MAX_HD>
__global__ void __launch_bounds__(WARPS * 32)
attention_simt_kernel(const T* __restrict__ qkv, T* __restrict__ out,
                      const T* __restrict__ k_pool, const T* __restrict__ v_pool,
                      const int* __restrict__ block_table, int max_blocks,
                      const int* __restrict__ positions, const int* __restrict__ req_of_token,
                      int n_tokens, int n_heads, int n_kv, int hd, int block_size, float scale,
                      int window, float softcap, long long n_pages,
                      const float* __restrict__ sink, const float* __restrict__ slopes,
                      int keep_first, long long out_stride, int chunk) {
    chain_release();
    chain_wait();
    __shared__ float q_s[WARPS][MAX_HD];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long unit = (long long)blockIdx.x * WARPS + warp;   // (token, head)
    if (unit >= (long long)n_tokens * n_heads) return;
    const int t = (int)(unit / n_heads), h = (int)(unit % n_heads);
    const int kvh = h / (n_heads / n_kv);
    const int r = req_of_token[t];
    const int p = positions[t];
    const int row_w = (n_heads + 2 * n_kv) * hd;

    const T* qp = qkv + (size_t)t * row_w + (size_t)h * hd;
    for (int i = lane; i < hd; i += 32) q_s[warp][i] = Elem<T>::load(qp + i);
    __syncwarp();

    const int j_lo = max(0, first_visible(p, window, chunk));
    const int* table = block_table + (size_t)r * max_blocks;
    const int nd = (hd + 31) / 32;

    float m = -INFINITY, l = 0.f;
    float acc[MAX_HD / 32];
#pragma unroll
    for (int i = 0; i < MAX_HD / 32; ++i) acc[i] = 0.f;

    const int keep = j_lo > 0 ? min(keep_first, j_lo) : 0;   // kept keys the window would hide
    const float slope = slopes ? slopes[h] : 0.f;
    for (int j0 = keep > 0 ? 0 : (j_lo / 32) * 32; j0 <= p; j0 += 32) {
        if (j0 >= keep && j0 + 32 <= j_lo) {          // past the kept keys: on to the window
            j0 = (j_lo / 32) * 32 - 32;
            continue;
        }
        const int j = j0 + lane;
        const bool valid = (j >= j_lo || j < keep) && j <= p;
        float s = -INFINITY;
        if (valid) {
            const int page = table[j / block_size];
            const T* kr = k_pool + (((size_t)kvh * n_pages + page) * block_size + j % block_size) * hd;
            s = dot_row(q_s[warp], kr, hd) * scale;
            if (slopes) s -= slope * (float)(p - j);
            if (softcap > 0.f) s = softcap * tanhf(s / softcap);
        }
        const float m_new = fmaxf(m, warp_max(s));
        const float pj = valid ? expf(s - m_new) : 0.f;
        const float corr = expf(m - m_new);       // m = -inf on the first chunk: exp(-inf) = 0
        l = l * corr + warp_sum(pj);
#pragma unroll
        for (int i = 0; i < MAX_HD / 32; ++i) acc[i] *= corr;
        for (int jj = 0; jj < 32; ++jj) {
            const int key = j0 + jj;
            if ((key < j_lo && key >= keep) || key > p) continue;        // uniform across the warp
            const float pk = __shfl_sync(0xffffffffu, pj, jj);
            const int page = table[key / block_size];
            const T* vr = v_pool + (((size_t)kvh * n_pages + page) * block_size + key % block_size) * hd;
#pragma unroll
            for (int i = 0; i < MAX_HD / 32; ++i) {
                const int dd = lane + 32 * i;
                if (i < nd && dd < hd) acc[i] = fmaf(pk, Elem<T>::load(vr + dd), acc[i]);
            }
        }
        m = m_new;
    }
    T* op = out + (size_t)t * out_stride + (size_t)h * hd;
    if (sink) l += expf(sink[h] - m);         // every token sees itself: m is a number
    const float inv = 1.0f / l;
#pragma unroll
    for (int i = 0; i < MAX_HD / 32; ++i) {
        const int dd = lane + 32 * i;
        if (i < nd && dd < hd) Elem<T>::store(op + dd, acc[i] * inv);
    }
}
}  // namespace

MLS_API int mls_attention_simt(const void* qkv, void* out, int dtype, const void* k_pool,
                               const void* v_pool, const int* block_table, int max_blocks,
                               const int* positions, const int* req_of_token, int n_tokens,
                               int n_heads, int n_kv, int hd, int block_size, float scale,
                               int window, float softcap, long long n_pages, const float* sink,
                               const float* slopes, int keep_first, long long out_stride,
                               int chunk, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (hd > MOST_HD || hd <= 0 || n_heads % n_kv) return MLS_ERR_UNSUPPORTED;
    if (out_stride <= 0) out_stride = (long long)n_heads * hd;
    const long long units = (long long)n_tokens * n_heads;
    const int blocks = (int)((units + WARPS - 1) / WARPS);
#define SIMT_GO(T, HD)                                                                            \
    MLS_LAUNCH((attention_simt_kernel<T, HD>), dim3(blocks), dim3(WARPS * 32), 0, stream,          \
               (const T*)qkv, (T*)out, (const T*)k_pool, (const T*)v_pool, block_table, max_blocks, \
               positions, req_of_token, n_tokens, n_heads, n_kv, hd, block_size, scale, window,    \
               softcap, n_pages, sink, slopes, keep_first, out_stride, window > 0 ? 0 : chunk)
    if (dtype == MLS_BF16) {
        if (hd <= 512) SIMT_GO(__nv_bfloat16, 512);
        else SIMT_GO(__nv_bfloat16, MOST_HD);
    } else {
        if (hd <= 512) SIMT_GO(float, 512);
        else SIMT_GO(float, MOST_HD);
    }
#undef SIMT_GO
    return launch_status();
}
