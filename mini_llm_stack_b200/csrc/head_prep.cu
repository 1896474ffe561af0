// Preparation of grouped-query attention without rotation: from the float32 projection row
// [.. q heads (e each) .. k heads (e each) .. v heads (f each) ..] of every token of a step
//
//   q_h <- (q_h + b_q) ;  k_g <- (k_g + b_k) ;  v_g <- (v_g + b_v) * v_scale      biases optional
//   q_h <- q_h / sqrt(mean(q_h^2) + eps) * w_q, k_g likewise with w_k           per head, optional;
//                                                                  the weights [e] serve all heads
//   q_h <- q_h * (1 + coef * ln(floor((p + 1) / every) + 1))      the query's temperature at
//                                                                  position p, optional
//   v <- (1 - lambda) v + lambda v_first           optional: v_first [T, all v entries], float32,
//                    are the step's values of an earlier layer, which that layer leaves there
//
// q goes to the row the attention kernels read ([T, q_width], head h at h * hd), k and v into
// the pages at the step's slots.  Heads are hd wide in both places: the entries past e (past
// f for the values) are zeros, which changes no score and leaves zeros in the outputs' extra
// entries.  The rest of a page that a request enters in this step is cleared.
//
// (mls_head_prep_store).  One block a token, one warp a head at a time; sums of squares in float32 in lane-stride
// order and five shuffles, so a token's values depend on nothing else in the batch.
//
// mls_head_conv_rope_store: the same for attention with rotation, from contiguous columns
// [q heads | k heads | v heads] of the float32 projection row.  A head of q and k may consist of
// several maps (of e entries each, one after the other).  For every channel, then every map:
//
//   u <- u + b ;  y_t = sum_j w[j] u_(t - taps + 1 + j), zeros before the sequence's start  (optional)
//   q, k <- y / sqrt(mean(y^2) + eps) * w_q (w_k)              per map, optional
//   entry i < dims/2 of a map turns with entry i + dims/2 by position * freq[i]; cosine and sine
//   are multiplied by `amplitude`                                                           optional
//
// A cached key row is a head's maps side by side, a query row holds one map in its place and
// zeros elsewhere: with maps M > 1 head h's map m is a query head of its own (row h * M + m),
// and its score against the cached row is that of its own map's key.  The convolution's last
// taps - 1 inputs of every request are a tail [taps - 1, channels] (float32, oldest first) in its
// state slot; mls_tail_update moves it on behind this kernel or, in a step of one token a request,
// this kernel does itself.  A warp a map (or value head) and run of tokens.  Which of two kernels
// and how many entries a lane takes depends on the model's sizes alone.
//
// mls_head_difference: what becomes of two maps' outputs a head, a warp a (token, head):
//   o = a1 - lambda a2 ;  o <- o / sqrt(mean(o^2) + eps) * mul ;  o <- o * sigmoid(gate)
#include "common.cuh"
#include "page_tail.cuh"
#include "row_pack.cuh"

namespace {
constexpr int HP_THREADS = 128;      // a block of a prompt's token
constexpr int HP_MAX_THREADS = 512;  // few tokens: up to a warp a head, so that no warp takes many in turn

template <typename T>
__global__ void __launch_bounds__(HP_MAX_THREADS)
head_prep_kernel(const float* __restrict__ proj, int proj_width, int q_col, int k_col, int v_col,
                 const float* __restrict__ b_q, const float* __restrict__ b_k,
                 const float* __restrict__ b_v, const float* __restrict__ w_q,
                 const float* __restrict__ w_k, float eps, float temp_coef, int temp_every,
                 float v_scale, float* __restrict__ v_first, int v_mode, float v_lambda,
                 const int* __restrict__ positions,
                 const int* __restrict__ slot_map, T* __restrict__ q_out, int q_width,
                 T* __restrict__ k_pool, T* __restrict__ v_pool, int block_size, int n_pages,
                 int n_tokens, int n_heads, int n_kv, int e, int f, int hd, int writes,
                 int* __restrict__ status) {
    chain_release();
    const int t = blockIdx.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5;
    int slot = -1, rest = 0;
    if (writes) {
        slot = slot_map[t];
        if (slot < 0 || slot >= n_pages * block_size) {
            if (threadIdx.x == 0 && status) atomicOr(status, MLS_STATUS_BAD_SLOT);
            slot = -1;
        } else {
            rest = page_tail_to_clear(slot_map, t, n_tokens, slot, block_size);
        }
    }
    float temp = 1.f;
    if (temp_every > 0)
        temp = 1.0f + temp_coef * logf((float)((positions[t] + 1) / temp_every + 1));
    chain_wait();
    const float* row = proj + (size_t)t * proj_width;
    const int units = n_heads + (writes ? 2 * n_kv : 0);
    for (int u = warp; u < units; u += n_warps) {
        // which head this is, where it comes from and where it goes
        const int kind = u < n_heads ? 0 : (u < n_heads + n_kv ? 1 : 2);
        const int head = kind == 0 ? u : (kind == 1 ? u - n_heads : u - n_heads - n_kv);
        const int width = kind == 2 ? f : e;
        const float* src = row + (kind == 0 ? q_col : kind == 1 ? k_col : v_col) + (size_t)head * width;
        const float* bias = kind == 0 ? b_q : kind == 1 ? b_k : b_v;
        if (bias) bias += (size_t)head * width;
        const float* w = kind == 0 ? w_q : kind == 1 ? w_k : nullptr;
        T* dst;
        if (kind == 0) {
            dst = q_out + (size_t)t * q_width + (size_t)head * hd;
        } else {
            if (slot < 0) continue;
            const int page = slot / block_size, off = slot - page * block_size;
            dst = (kind == 1 ? k_pool : v_pool) +
                  (((size_t)head * n_pages + page) * block_size + off) * hd;
        }
        float mul = kind == 0 ? temp : (kind == 2 ? v_scale : 1.f);
        if (w) {
            float ss = 0.f;
            for (int i = lane; i < width; i += 32) {
                const float x = src[i] + (bias ? bias[i] : 0.f);
                ss = fmaf(x, x, ss);
            }
            mul *= 1.0f / sqrtf(warp_sum(ss) / (float)width + eps);
        }
        for (int i = lane; i < hd; i += 32) {
            float x = 0.f;
            if (i < width) {
                x = (src[i] + (bias ? bias[i] : 0.f)) * mul;
                if (w) x *= w[i];
                if (kind == 2 && v_mode != 0) {
                    float* first = v_first + ((size_t)t * n_kv + head) * f + i;
                    if (v_mode == 1) *first = x;
                    else x = (1.0f - v_lambda) * x + v_lambda * *first;
                }
            }
            Elem<T>::store(dst + i, x);
        }
    }
    if (writes && slot >= 0) {
        __syncthreads();
        clear_page_tail<T>(rest, slot, block_size, n_pages, n_kv, hd, k_pool, v_pool);
    }
}

constexpr int HC_WARPS = 8, HC_RUN = 8, HC_TAPS = 8;

struct HeadConvArgs {
    const float* proj;                 // [T, proj_width], q | k | v from column col on
    int proj_width, col;
    const float* bias;                 // [channels] or nullptr
    const float* conv;                 // [taps][channels], taps > 0
    int taps, move_tail;
    float* tail;                       // [slots][taps - 1][channels], tail_stride apart
    long long tail_stride;
    const float *w_q, *w_k;            // [e] or nullptr
    float eps;
    const double* freq;                // [rot / 2]
    int rot;
    float amplitude;
    const int *state_slot, *cu_q, *req_of_token, *positions, *slot_map;
    int q_width, block_size, n_pages, n_tokens, n_heads, n_kv, maps, e, f, hd, writes, run;
    int* status;
};

template <int V>
__device__ __forceinline__ Pack<V> load_floats(const float* p) {
    Pack<V> r;
    if constexpr (V == 4) {
        const float4 x = *reinterpret_cast<const float4*>(p);
        r.v[0] = x.x; r.v[1] = x.y; r.v[2] = x.z; r.v[3] = x.w;
    } else if constexpr (V == 2) {
        const float2 x = *reinterpret_cast<const float2*>(p);
        r.v[0] = x.x; r.v[1] = x.y;
    } else {
        r.v[0] = *p;
    }
    return r;
}
template <int V>
__device__ __forceinline__ void store_floats(float* p, const Pack<V>& r) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else if constexpr (V == 2) *reinterpret_cast<float2*>(p) = make_float2(r.v[0], r.v[1]);
    else *p = r.v[0];
}
template <int V>
__device__ __forceinline__ void store_elems(float* p, const Pack<V>& r) { store_floats<V>(p, r); }
template <int V>
__device__ __forceinline__ void store_elems(__nv_bfloat16* p, const Pack<V>& r) {
    if constexpr (V == 4)
        *reinterpret_cast<uint2*>(p) = pack_bf16x4(make_float4(r.v[0], r.v[1], r.v[2], r.v[3]));
    else if constexpr (V == 2)
        *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(r.v[0], r.v[1]);
    else
        *p = __float2bfloat16_rn(r.v[0]);
}

// What the kernels below look up once for a run of tokens: each token's cache slot (-1: none), the
// slots behind it to clear, its place among its request's tokens of this step and its request's
// state slot; and the angles' cosines and sines.  All of it is the step's own input, which no kernel
// of the step writes.
struct RunTokens {
    int slot[HC_RUN], rest[HC_RUN], at[HC_RUN], state[HC_RUN];
};
__device__ __forceinline__ void look_up_run(const HeadConvArgs& a, int t0, int n_run, RunTokens& R,
                                            float* angles) {
    const int half = a.rot / 2;
    if (threadIdx.x < n_run) {
        const int t = t0 + threadIdx.x, r = a.req_of_token[t];
        int slot = -1, rest = 0;
        if (a.writes) {
            slot = a.slot_map[t];
            if (slot < 0 || slot >= a.n_pages * a.block_size) {
                if (blockIdx.y == 0 && a.status) atomicOr(a.status, MLS_STATUS_BAD_SLOT);
                slot = -1;
            } else {
                rest = page_tail_to_clear(a.slot_map, t, a.n_tokens, slot, a.block_size);
            }
        }
        R.slot[threadIdx.x] = slot;
        R.rest[threadIdx.x] = rest;
        R.at[threadIdx.x] = t - a.cu_q[r];
        R.state[threadIdx.x] = a.taps > 1 ? a.state_slot[r] : 0;
    }
    for (int u = threadIdx.x; u < n_run * half; u += blockDim.x) {
        const int tok = u / half, i = u - tok * half;
        float c, s;
        angle_cos_sin(a.positions[t0 + tok], a.freq[i], c, s);
        angles[tok * a.rot + i] = c * a.amplitude;
        angles[tok * a.rot + half + i] = s * a.amplitude;
    }
    __syncthreads();
}
template <typename T>
__device__ __forceinline__ void clear_run_tails(const HeadConvArgs& a, int n_run, const RunTokens& R,
                                                T* k_pool, T* v_pool) {
    if (!a.writes || blockIdx.y != 0) return;
    for (int tok = 0; tok < n_run; ++tok)
        if (R.slot[tok] >= 0)
            clear_page_tail<T>(R.rest[tok], R.slot[tok], a.block_size, a.n_pages, a.n_kv, a.hd, k_pool,
                               v_pool);
}

// V: neighbouring entries a lane takes at a time (the model's sizes decide).
template <typename T, int V>
__global__ void __launch_bounds__(HC_WARPS * 32)
head_conv_rope_kernel(const HeadConvArgs a, T* __restrict__ q_out, T* __restrict__ k_pool,
                      T* __restrict__ v_pool) {
    chain_release();
    extern __shared__ __align__(16) float hc_smem[];
    __shared__ RunTokens R;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t0 = blockIdx.x * a.run, n_run = min(a.run, a.n_tokens - t0);
    const int half = a.rot / 2, widest = max(a.e, a.f);
    float* angles = hc_smem;                                     // [run][cos | sin]
    float* stage = hc_smem + (((size_t)a.run * a.rot + 3) & ~(size_t)3) +
                   (size_t)warp * ((widest + 3) & ~3);           // this warp's head
    look_up_run(a, t0, n_run, R, angles);
    chain_wait();
    const int nq = a.n_heads * a.maps, nk = a.n_kv * a.maps;
    const int units = nq + (a.writes ? nk + a.n_kv : 0);
    const int channels = (nq + nk) * a.e + a.n_kv * a.f, n_tail = a.taps - 1;
    const int u = blockIdx.y * HC_WARPS + warp;
    if (u < units) {
        const int kind = u < nq ? 0 : (u < nq + nk ? 1 : 2);
        const int unit = kind == 0 ? u : (kind == 1 ? u - nq : u - nq - nk);
        const int width = kind == 2 ? a.f : a.e;
        const int ch0 = kind == 2 ? (nq + nk) * a.e + unit * a.f : u * a.e;    // first channel
        const float* w = kind == 0 ? a.w_q : kind == 1 ? a.w_k : nullptr;
        const int head = kind == 2 ? unit : unit / a.maps, map = kind == 2 ? 0 : unit % a.maps;
        const int inside = map * a.e;                            // where the map lies in its row
        const int rot = kind == 2 ? 0 : a.rot;
        // the entries of the row this warp writes: a query row is its own; a key row's maps share
        // one, the last of them fills it up
        const int c_lo = kind == 1 ? inside : 0;
        const int c_hi = (kind == 1 && map + 1 < a.maps) ? inside + a.e : a.hd;
        for (int tok = 0; tok < n_run; ++tok) {
            const int t = t0 + tok, i_t = R.at[tok];
            float* tail = n_tail > 0 ? a.tail + (size_t)R.state[tok] * a.tail_stride : nullptr;
            float ss = 0.f;
            for (int c = lane * V; c < width; c += 32 * V) {
                const int ch = ch0 + c;
                const float* src = a.proj + (size_t)t * a.proj_width + a.col + ch;
                Pack<V> bias;
#pragma unroll
                for (int x = 0; x < V; ++x) bias.v[x] = 0.f;
                if (a.bias) bias = load_floats<V>(a.bias + ch);
                Pack<V> y;
                if (a.taps <= 0) {
                    y = load_floats<V>(src);
#pragma unroll
                    for (int x = 0; x < V; ++x) y.v[x] += bias.v[x];
                } else {
#pragma unroll
                    for (int x = 0; x < V; ++x) y.v[x] = 0.f;
                    for (int j0 = 0; j0 < a.taps; j0 += HC_TAPS) {
                        Pack<V> in[HC_TAPS];
#pragma unroll
                        for (int j = 0; j < HC_TAPS; ++j) {
                            const int back = n_tail - (j0 + j);      // tokens before this one
                            if (j0 + j < a.taps)
                                in[j] = back <= i_t
                                    ? load_floats<V>(src - (size_t)back * a.proj_width)
                                    : load_floats<V>(tail + (size_t)(n_tail + i_t - back) * channels + ch);
                        }
#pragma unroll
                        for (int j = 0; j < HC_TAPS; ++j) {
                            if (j0 + j < a.taps) {
                                if (n_tail - (j0 + j) <= i_t) {
#pragma unroll
                                    for (int x = 0; x < V; ++x) in[j].v[x] += bias.v[x];
                                }
                                const Pack<V> cw = load_floats<V>(a.conv + (size_t)(j0 + j) * channels + ch);
#pragma unroll
                                for (int x = 0; x < V; ++x) y.v[x] = fmaf(cw.v[x], in[j].v[x], y.v[x]);
                                // (row j - 1 was read by this lane one tap ago)
                                if (a.move_tail && j0 + j >= 1)
                                    store_floats<V>(tail + (size_t)(j0 + j - 1) * channels + ch, in[j]);
                            }
                        }
                    }
                }
                if (w) {
                    const Pack<V> wv = load_floats<V>(w + c);
#pragma unroll
                    for (int x = 0; x < V; ++x) {
                        ss = fmaf(y.v[x], y.v[x], ss);
                        y.v[x] *= wv.v[x];
                    }
                }
                store_floats<V>(stage + c, y);
            }
            const float inv = w ? 1.0f / sqrtf(warp_sum(ss) / (float)width + a.eps) : 1.f;
            __syncwarp();
            T* dst;
            if (kind == 0) {
                dst = q_out + (size_t)t * a.q_width + (size_t)unit * a.hd;
            } else {
                const int slot = R.slot[tok];
                if (slot < 0) continue;                          // (the same for the whole warp)
                const int page = slot / a.block_size, off = slot - page * a.block_size;
                dst = (kind == 1 ? k_pool : v_pool) +
                      (((size_t)head * a.n_pages + page) * a.block_size + off) * a.hd;
            }
            const float* cs = angles + tok * a.rot;
            for (int c = c_lo + lane * V; c < c_hi; c += 32 * V) {
                const int rel = c - inside;
                Pack<V> y;
#pragma unroll
                for (int x = 0; x < V; ++x) {
                    const int i = rel + x;
                    float val = 0.f;
                    if (i >= 0 && i < width) {
                        val = stage[i] * inv;
                        if (i < half && rot > 0) {
                            const float mate = stage[i + half] * inv;
                            val = __fsub_rn(__fmul_rn(val, cs[i]), __fmul_rn(mate, cs[half + i]));
                        } else if (i < rot) {
                            const float mate = stage[i - half] * inv;
                            val = __fadd_rn(__fmul_rn(val, cs[i - half]), __fmul_rn(mate, cs[i]));
                        }
                    }
                    y.v[x] = val;
                }
                store_elems<V>(dst + c, y);
            }
            __syncwarp();                                        // the stage is filled again
        }
    }
    clear_run_tails<T>(a, n_run, R, k_pool, v_pool);
}

// The same with a lane's entries in registers: a lane takes V entries and the V that turn with
// them (past the rotated ones: the V behind them), so a map or value head of up to 64 V entries
// needs at most a warp, a smaller one a power of two of lanes, and a warp works on as many tokens
// of the run at a time as fit it.  TAPS: 0, or the most taps (weights, biases and norm weights are
// then read once a run).
template <typename T, int V, int TAPS>
__global__ void __launch_bounds__(HC_WARPS * 32, V == 4 ? 2 : 3)
head_conv_rope_lanes_kernel(const HeadConvArgs a, T* __restrict__ q_out, T* __restrict__ k_pool,
                            T* __restrict__ v_pool) {
    chain_release();
    extern __shared__ __align__(16) float hc_smem[];
    __shared__ RunTokens R;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t0 = blockIdx.x * a.run, n_run = min(a.run, a.n_tokens - t0);
    const int half = a.rot / 2;
    float* angles = hc_smem;
    look_up_run(a, t0, n_run, R, angles);
    const int nq = a.n_heads * a.maps, nk = a.n_kv * a.maps;
    const int units = nq + (a.writes ? nk + a.n_kv : 0);
    const int channels = (nq + nk) * a.e + a.n_kv * a.f, n_tail = a.taps - 1;
    const int u = blockIdx.y * HC_WARPS + warp;
    const bool there = u < units;
    const int kind = u < nq ? 0 : (u < nq + nk ? 1 : 2);
    const int unit = kind == 0 ? u : (kind == 1 ? u - nq : u - nq - nk);
    const int width = kind == 2 ? a.f : a.e;
    const int ch0 = kind == 2 ? (nq + nk) * a.e + unit * a.f : u * a.e;
    const float* w = kind == 0 ? a.w_q : kind == 1 ? a.w_k : nullptr;
    const int head = kind == 2 ? unit : unit / a.maps, map = kind == 2 ? 0 : unit % a.maps;
    const int inside = map * a.e, rot = kind == 2 ? 0 : a.rot;
    const int turning = rot / (2 * V);                           // lanes whose entries turn
    const int items = turning + ((width - rot) / V + 1) / 2;
    int lanes = 1;
    while (lanes < items) lanes <<= 1;                           // (at most 32: the host's choice)
    const int at_once = 32 / lanes, mine = lane & (lanes - 1), group = lane / lanes;
    const bool turns = mine < turning;
    const int ca = turns ? mine * V : rot + (mine - turning) * 2 * V;      // this lane's entries
    const int cb = turns ? ca + half : ca + V;
    const bool has_a = there && mine < items, has_b = has_a && cb < width;
    // the rest of the row that this warp fills with zeros
    const int z_lo = kind == 2 ? width : (kind == 1 ? (map + 1 < a.maps ? a.hd : a.maps * a.e) : 0);

    Pack<V> bias[2], cw[2][TAPS > 0 ? TAPS : 1], wv[2];
#pragma unroll
    for (int x = 0; x < 2; ++x) {
        const int c = x ? cb : ca;
        const bool has = x ? has_b : has_a;
#pragma unroll
        for (int k = 0; k < V; ++k) {
            bias[x].v[k] = 0.f;
            wv[x].v[k] = 1.f;
        }
        if (has && a.bias) bias[x] = load_floats<V>(a.bias + ch0 + c);
        if (has && w) wv[x] = load_floats<V>(w + c);
        if constexpr (TAPS > 0) {
#pragma unroll
            for (int j = 0; j < TAPS; ++j)
                if (has && j < a.taps)
                    cw[x][j] = load_floats<V>(a.conv + (size_t)j * channels + ch0 + c);
        }
    }
    chain_wait();
    for (int tok0 = 0; tok0 < n_run; tok0 += at_once) {
        const int tok = tok0 + group, t = t0 + tok;
        const bool live = tok < n_run;
        Pack<V> y[2];
        float ss = 0.f;
        const int i_t = live ? R.at[tok] : 0;
        float* tail = (live && n_tail > 0) ? a.tail + (size_t)R.state[tok] * a.tail_stride : nullptr;
#pragma unroll
        for (int x = 0; x < 2; ++x) {
#pragma unroll
            for (int k = 0; k < V; ++k) y[x].v[k] = 0.f;
            if (!live || !(x ? has_b : has_a)) continue;
            const int ch = ch0 + (x ? cb : ca);
            const float* src = a.proj + (size_t)t * a.proj_width + a.col + ch;
            if constexpr (TAPS == 0) {
                y[x] = load_floats<V>(src);
#pragma unroll
                for (int k = 0; k < V; ++k) y[x].v[k] += bias[x].v[k];
            } else {
                Pack<V> in[TAPS];
#pragma unroll
                for (int j = 0; j < TAPS; ++j) {
                    const int back = n_tail - j;                 // tokens before this one
                    if (j < a.taps)
                        in[j] = back <= i_t
                            ? load_floats<V>(src - (size_t)back * a.proj_width)
                            : load_floats<V>(tail + (size_t)(n_tail + i_t - back) * channels + ch);
                }
#pragma unroll
                for (int j = 0; j < TAPS; ++j) {
                    if (j < a.taps) {
                        if (n_tail - j <= i_t) {
#pragma unroll
                            for (int k = 0; k < V; ++k) in[j].v[k] += bias[x].v[k];
                        }
#pragma unroll
                        for (int k = 0; k < V; ++k)
                            y[x].v[k] = fmaf(cw[x][j].v[k], in[j].v[k], y[x].v[k]);
                        if (a.move_tail && j >= 1)
                            store_floats<V>(tail + (size_t)(j - 1) * channels + ch, in[j]);
                    }
                }
            }
#pragma unroll
            for (int k = 0; k < V; ++k) ss = fmaf(y[x].v[k], y[x].v[k], ss);
        }
        if (w) {
            for (int o = lanes >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            const float inv = 1.0f / sqrtf(ss / (float)width + a.eps);
#pragma unroll
            for (int x = 0; x < 2; ++x)
#pragma unroll
                for (int k = 0; k < V; ++k) y[x].v[k] = y[x].v[k] * inv * wv[x].v[k];
        }
        if (!live || !there) continue;
        if (turns) {
            const Pack<V> c = load_floats<V>(angles + tok * a.rot + ca);
            const Pack<V> s = load_floats<V>(angles + tok * a.rot + half + ca);
#pragma unroll
            for (int k = 0; k < V; ++k) {
                const float p = y[0].v[k], q = y[1].v[k];
                y[0].v[k] = __fsub_rn(__fmul_rn(p, c.v[k]), __fmul_rn(q, s.v[k]));
                y[1].v[k] = __fadd_rn(__fmul_rn(q, c.v[k]), __fmul_rn(p, s.v[k]));
            }
        }
        T* dst;
        if (kind == 0) {
            dst = q_out + (size_t)t * a.q_width + (size_t)unit * a.hd;
        } else {
            const int slot = R.slot[tok];
            if (slot < 0) continue;
            const int page = slot / a.block_size, off = slot - page * a.block_size;
            dst = (kind == 1 ? k_pool : v_pool) +
                  (((size_t)head * a.n_pages + page) * a.block_size + off) * a.hd;
        }
        if (has_a) store_elems<V>(dst + inside + ca, y[0]);
        if (has_b) store_elems<V>(dst + inside + cb, y[1]);
        Pack<V> zero;
#pragma unroll
        for (int k = 0; k < V; ++k) zero.v[k] = 0.f;
        for (int z = z_lo + mine * V; z < a.hd; z += lanes * V)
            if (kind != 0 || z < inside || z >= inside + a.e) store_elems<V>(dst + z, zero);
    }
    clear_run_tails<T>(a, n_run, R, k_pool, v_pool);
}

// o [T, 2 H * hd]: head h's two maps at rows 2h and 2h + 1; out [T, H * f].
template <typename T, int V>
__global__ void __launch_bounds__(256)
head_difference_kernel(const T* __restrict__ o, int hd, float lambda, float mul, float eps,
                       const float* __restrict__ gate, int gate_row, int gate_col,
                       T* __restrict__ out, int n_tokens, int n_heads, int f) {
    chain_release();
    chain_wait();
    const int lane = threadIdx.x & 31;
    const long long unit = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (unit >= (long long)n_tokens * n_heads) return;
    const int t = (int)(unit / n_heads), h = (int)(unit - (long long)t * n_heads);
    constexpr int DT = sizeof(T) == 2 ? MLS_BF16 : MLS_F32;
    const size_t first = ((size_t)t * n_heads + h) * 2 * hd;
    auto difference = [&](int c) {
        const Pack<V> a1 = load_pack<V>(o, first + c, DT), a2 = load_pack<V>(o, first + hd + c, DT);
        Pack<V> r;
#pragma unroll
        for (int x = 0; x < V; ++x) r.v[x] = fmaf(-lambda, a2.v[x], a1.v[x]);
        return r;
    };
    float ss = 0.f;
    for (int c = lane * V; c < f; c += 32 * V) {
        const Pack<V> d = difference(c);
#pragma unroll
        for (int x = 0; x < V; ++x) ss = fmaf(d.v[x], d.v[x], ss);
    }
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)f + eps);
    for (int c = lane * V; c < f; c += 32 * V) {
        Pack<V> d = difference(c);
        Pack<V> z;
        if (gate) z = load_pack<V>(gate, (size_t)t * gate_row + gate_col + (size_t)h * f + c, MLS_F32);
#pragma unroll
        for (int x = 0; x < V; ++x) {
            d.v[x] = d.v[x] * inv * mul;
            if (gate) d.v[x] = d.v[x] / (1.0f + expf(-z.v[x]));
        }
        store_pack<V>(out, ((size_t)t * n_heads + h) * f + c, DT, d);
    }
}
}  // namespace

MLS_API int mls_head_prep_store(const float* proj, int proj_width, int q_col, int k_col, int v_col,
                                const float* b_q, const float* b_k, const float* b_v,
                                const float* w_q, const float* w_k, float eps, float temp_coef,
                                int temp_every, float v_scale, float* v_first, int v_mode,
                                float v_lambda, const int* positions,
                                const int* slot_map, void* q_out, int q_width, int dtype,
                                void* k_pool, void* v_pool, int block_size, int n_pages,
                                int n_tokens, int n_heads, int n_kv, int e, int f, int hd,
                                int writes, int* status, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (e <= 0 || f <= 0 || hd < e || hd < f || n_heads <= 0 || n_kv <= 0 ||
        v_mode < 0 || v_mode > 2 || (v_mode && (!v_first || !writes)))
        return MLS_ERR_UNSUPPORTED;
    const int units = n_heads + (writes ? 2 * n_kv : 0);
    const int threads = n_tokens > 64 ? HP_THREADS
        : (32 * units < HP_THREADS ? HP_THREADS : (32 * units > HP_MAX_THREADS ? HP_MAX_THREADS : 32 * units));
    if (dtype == MLS_BF16)
        MLS_LAUNCH((head_prep_kernel<__nv_bfloat16>), dim3(n_tokens), dim3(threads), 0, stream,
                   proj, proj_width, q_col, k_col, v_col, b_q, b_k, b_v, w_q, w_k, eps, temp_coef,
                   temp_every, v_scale, v_first, v_mode, v_lambda, positions, slot_map, (__nv_bfloat16*)q_out, q_width,
                   (__nv_bfloat16*)k_pool, (__nv_bfloat16*)v_pool, block_size, n_pages, n_tokens,
                   n_heads, n_kv, e, f, hd, writes, status);
    else
        MLS_LAUNCH((head_prep_kernel<float>), dim3(n_tokens), dim3(threads), 0, stream, proj,
                   proj_width, q_col, k_col, v_col, b_q, b_k, b_v, w_q, w_k, eps, temp_coef,
                   temp_every, v_scale, v_first, v_mode, v_lambda, positions, slot_map, (float*)q_out, q_width,
                   (float*)k_pool, (float*)v_pool, block_size, n_pages, n_tokens, n_heads, n_kv,
                   e, f, hd, writes, status);
    return launch_status();
}

MLS_API int mls_head_conv_rope_store(
        const float* proj, int proj_width, int col, const float* bias, const float* conv, int taps,
        int move_tail, float* tail, long long tail_stride, const float* w_q, const float* w_k,
        float eps, const double* freq, int rot, float amplitude, const int* state_slot,
        const int* cu_q, const int* req_of_token, const int* positions, const int* slot_map,
        void* q_out, int q_width, int dtype, void* k_pool, void* v_pool, int block_size, int n_pages,
        int n_tokens, int n_heads, int n_kv, int maps, int e, int f, int hd, int writes, int* status,
        cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (e <= 0 || f <= 0 || maps < 1 || hd < maps * e || hd < f || n_heads <= 0 || n_kv <= 0 ||
        taps < 0 || (taps > 0 && !conv) || (taps > 1 && !tail) || rot < 0 || (rot & 1) || rot > e ||
        (rot > 0 && !freq) || (w_q == nullptr) != (w_k == nullptr) || (move_tail && taps <= 1))
        return MLS_ERR_UNSUPPORTED;
    HeadConvArgs a;
    a.proj = proj; a.proj_width = proj_width; a.col = col; a.bias = bias; a.conv = conv; a.taps = taps;
    a.move_tail = move_tail; a.tail = tail; a.tail_stride = tail_stride; a.w_q = w_q; a.w_k = w_k;
    a.eps = eps; a.freq = freq; a.rot = rot; a.amplitude = amplitude; a.state_slot = state_slot;
    a.cu_q = cu_q; a.req_of_token = req_of_token; a.positions = positions; a.slot_map = slot_map;
    a.q_width = q_width; a.block_size = block_size; a.n_pages = n_pages; a.n_tokens = n_tokens;
    a.n_heads = n_heads; a.n_kv = n_kv; a.maps = maps; a.e = e; a.f = f; a.hd = hd; a.writes = writes;
    a.status = status;
    const int units = n_heads * maps + (writes ? n_kv * maps + n_kv : 0);
    const int grid_y = (units + HC_WARPS - 1) / HC_WARPS;
    // runs of tokens as long as every SM still has several blocks
    a.run = HC_RUN;
    while (a.run > 1 && (long long)((n_tokens + a.run - 1) / a.run) * grid_y < 4LL * sm_count())
        a.run >>= 1;
    // entries a lane takes at a time: all lanes busy, and every row at an aligned place
    const int widest = e > f ? e : f;
    auto takes = [&](int v) {
        uintptr_t bits = 0;
        for (const void* p : {(const void*)proj, (const void*)bias, (const void*)conv,
                              (const void*)tail, (const void*)w_q, (const void*)w_k})
            bits |= reinterpret_cast<uintptr_t>(p);
        return e % v == 0 && f % v == 0 && proj_width % v == 0 && col % v == 0 && q_width % v == 0 &&
               bits % (4 * v) == 0 && (taps <= 1 || tail_stride % v == 0);
    };
    // with the entries in registers where a map (a value head) fits a warp and the taps their array
    int v = takes(4) && rot % 8 == 0 ? 4 : takes(2) && rot % 4 == 0 ? 2 : 1;
    auto items = [&](int width, int turned) { return turned / (2 * v) + ((width - turned) / v + 1) / 2; };
    const bool lanes = taps <= 4 && items(e, rot) <= 32 && items(f, 0) <= 32;
    if (!lanes) v = (widest > 64 && takes(4)) ? 4 : (widest > 32 && takes(2)) ? 2 : 1;
    const size_t smem = ((((size_t)a.run * rot + 3) & ~(size_t)3) +
                         (lanes ? 0 : (size_t)HC_WARPS * ((widest + 3) & ~3))) * sizeof(float);
    if (smem > 48 * 1024) return MLS_ERR_UNSUPPORTED;
    const dim3 grid((n_tokens + a.run - 1) / a.run, grid_y);
#define HC_RUN_KERNEL(K)                                                                          \
    MLS_LAUNCH(K, grid, dim3(HC_WARPS * 32), smem, stream, a, (E*)q_out, (E*)k_pool, (E*)v_pool)
#define HC_GO(V)                                                                                  \
    do {                                                                                          \
        if (!lanes) HC_RUN_KERNEL((head_conv_rope_kernel<E, V>));                                 \
        else if (taps > 0) HC_RUN_KERNEL((head_conv_rope_lanes_kernel<E, V, 4>));                 \
        else HC_RUN_KERNEL((head_conv_rope_lanes_kernel<E, V, 0>));                               \
    } while (0)
#define HC_TYPE(TYPE)                                                                             \
    do {                                                                                          \
        using E = TYPE;                                                                           \
        if (v == 4) HC_GO(4);                                                                     \
        else if (v == 2) HC_GO(2);                                                                \
        else HC_GO(1);                                                                            \
    } while (0)
    if (dtype == MLS_BF16) HC_TYPE(__nv_bfloat16);
    else HC_TYPE(float);
#undef HC_TYPE
#undef HC_GO
#undef HC_RUN_KERNEL
    return launch_status();
}

MLS_API int mls_head_difference(const void* o, int dtype, int hd, float lambda, float mul, float eps,
                                const float* gate, int gate_row, int gate_col, void* out,
                                int n_tokens, int n_heads, int f, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (f <= 0 || hd < f || n_heads <= 0) return MLS_ERR_UNSUPPORTED;
    const int blocks = (int)(((long long)n_tokens * n_heads + 7) / 8);
    const bool by4 = f % 4 == 0 && hd % 4 == 0 && gate_row % 4 == 0 && gate_col % 4 == 0 &&
                     (reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(out) |
                      reinterpret_cast<uintptr_t>(gate)) % 16 == 0;
#define HD_GO(T, V)                                                                               \
    MLS_LAUNCH((head_difference_kernel<T, V>), dim3(blocks), dim3(256), 0, stream, (const T*)o, hd, \
               lambda, mul, eps, gate, gate_row, gate_col, (T*)out, n_tokens, n_heads, f)
    if (dtype == MLS_BF16) {
        if (by4) HD_GO(__nv_bfloat16, 4);
        else HD_GO(__nv_bfloat16, 1);
    } else {
        if (by4) HD_GO(float, 4);
        else HD_GO(float, 1);
    }
#undef HD_GO
    return launch_status();
}
