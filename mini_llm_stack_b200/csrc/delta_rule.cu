// The gated delta rule: a matrix state per head that decays, forgets what it holds under the
// token's key and takes the token's value in, carried from token to token in a float32 state
// slot per request.
//
// Per head, with key size e, value size f, state S [e, f], unit vectors q (times e^-1/2) and k,
// a decay g in (0, 1) and a step size b in (0, 1) per token:
//
//   S <- g S;   u = b (v - S^T k);   S <- S + k u^T;   o = S^T q
//
// q, k and v are projections that pass a short causal convolution per channel and silu; several
// value heads may share a key head.  Written with the state before the token, the token needs
// two products with it that do not wait for one another, S^T k and S^T q:
//
//   u = b (v - g S^T k);   o = g S^T q + (k . q) u;   S <- g S + k u^T
//
//   mls_delta_prep   projection rows (float32) -> convolution, silu, unit vectors, k . q, decay
//                    and step size, as the rows the scan reads
//   mls_delta_scan   walks the tokens of every request through the state; also stores the
//                    convolution's last inputs
//   mls_delta_step   one token a request: all of the above and what follows (norm over the
//                    head's values, weight, silu gate) in one kernel
//
// Layout of a request's state slot: S of every head transposed and padded, [H][fr][er] with
// er = e rounded up to 32 and fr = f rounded up to 16 (the padding stays zero), then the
// convolution's inputs as a ring [taps][channels]: position p lies in row p mod taps, so a
// token's row never falls on a row that its own convolution reads.  Rows of positions before
// the sequence's start are never read.
//
// A warp owns columns of S with eight lanes a column; a lane keeps er / 8 rows of each of its
// columns in registers, four neighbouring rows at a time (16-byte accesses of the state and of
// k and q), and multiplies them two at a time (fma.rn.f32x2).  The sum over the rows is the
// lane's own in a fixed order and three shuffles: a token's bits do not depend on the batch.
// The scan takes two tokens at a time from a portion's start, which moves the last bits where
// a cut separates two tokens.  Everything is float32.
#include "common.cuh"
#include "tma.cuh"

namespace {
constexpr float DR_UNIT_EPS = 1e-6f;     // inside the root of the unit vectors

__device__ __forceinline__ float silu1(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float sigmoid1(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus1(float z) {
    return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
}

// Two float32 operations in one instruction on register pairs.
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack2(float a, float b) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ float sum2(f32x2 v) {
    float a, b;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v));
    return a + b;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
    f32x2 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ f32x2 add2(f32x2 a, f32x2 b) {
    f32x2 d;
    asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
// the sum over the eight lanes that share a column
__device__ __forceinline__ float column_sum(float v) {
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    v += __shfl_xor_sync(0xffffffffu, v, 2);
    v += __shfl_xor_sync(0xffffffffu, v, 4);
    return v;
}
// Sizes, places and parameters every kernel here needs.
struct DeltaArgs {
    const float* proj;                 // [parts][T, width]: q heads | k heads | v heads, gates, ...
    int n_parts;
    long long part_stride;
    int width, qkv_col, a_col, b_col, g_col;
    const void* conv;                  // [channels, taps], last column meets the current token
    int conv_dtype, taps, channels;    // channels = 2 G e + H f, in the order of the projection
    const float* a_exp;                // [H]: exp(A_log)
    const float* dt_bias;              // [H]
    const int* state_slot;
    const int* cu_q;
    const int* req_of_token;
    const int* positions;
    float* state;                      // [slots], state_stride floats apart
    long long state_stride, ring_at;   // ring_at: the ring's place in a slot
    int n_tokens, n_requests;
    int H, G, e, f, er, fr;
    float q_scale;                     // e^-1/2
    __device__ __forceinline__ float at(int t, int col) const {
        const float* p = proj + (size_t)t * width + col;
        float s = *p;
        int k = 1;
        for (; k + 4 <= n_parts; k += 4) {
            float w[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) w[i] = p[(size_t)(k + i) * part_stride];
#pragma unroll
            for (int i = 0; i < 4; ++i) s += w[i];
        }
        for (; k < n_parts; ++k) s += p[(size_t)k * part_stride];
        return s;
    }
    __device__ __forceinline__ float* ring(int slot) const {
        return state + (size_t)slot * state_stride + ring_at;
    }
};

// What the scan reads, float32, so that the tokens of a pass are one run of memory each:
//   [G][T][q: er | k: er]      [H][fr / 16][T][16 values]      [H][T][DR_SCALARS]
// with the scalars of a value head and token: decay, step, k . q, k' . k, k' . q, 0, 0, 0, where k'
// is the key of the token before (anything where a request's tokens of the step begin).
constexpr int DR_SCALARS = 8, DR_COLS = 16;
struct Prepared {
    size_t v_at, s_at;                 // where the values and the scalars begin
    size_t T;
    int er, fr;
    __host__ __device__ Prepared(int n_tokens, int H, int G, int er_, int fr_)
        : v_at((size_t)n_tokens * G * 2 * er_), s_at(v_at + (size_t)n_tokens * H * fr_),
          T((size_t)n_tokens), er(er_), fr(fr_) {}
    __host__ __device__ size_t qk(int kv, int t) const { return ((size_t)kv * T + t) * 2 * er; }
    __host__ __device__ size_t v(int head, int chunk, int t) const {
        return v_at + (((size_t)head * (fr / DR_COLS) + chunk) * T + t) * DR_COLS;
    }
    __host__ __device__ size_t scalars(int head, int t) const {
        return s_at + ((size_t)head * T + t) * DR_SCALARS;
    }
};
__host__ __device__ inline int prepared_floats(int H, int G, int er, int fr) {      // a token's share
    return 2 * G * er + H * (fr + DR_SCALARS);
}

// A head's channels spread over a warp (channel lane + 32 i) with the convolution's weights and
// its last inputs; TT >= taps, the places before the real taps count as zero.
template <int NI, int TT>
struct ConvHead {
    float w[TT][NI], win[TT - 1][NI];
    int col, first, n;                 // column in a projection row, first channel, channels
    __device__ __forceinline__ void init(const DeltaArgs& a, int channel0, int count, int lane) {
        col = a.qkv_col + channel0;
        first = channel0;
        n = count;
#pragma unroll
        for (int j = 0; j < TT; ++j)
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const int c = lane + 32 * i, tap = j - (TT - a.taps);
                w[j][i] = (tap >= 0 && c < n)
                    ? load_as_float(a.conv, (size_t)(first + c) * a.taps + tap, a.conv_dtype) : 0.f;
            }
    }
    // the inputs before token t (the i_t-th of this step of its request, at position p)
    __device__ __forceinline__ void fill(const DeltaArgs& a, int t, int i_t, int p,
                                         const float* ring, int lane) {
#pragma unroll
        for (int j = 0; j < TT - 1; ++j) {
            const int back = TT - 1 - j;
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const int c = lane + 32 * i;
                float v = 0.f;
                if (back < a.taps && back <= p && c < n)
                    v = back <= i_t ? a.proj[(size_t)(t - back) * a.width + col + c]
                                    : ring[(size_t)((p - back) % a.taps) * a.channels + first + c];
                win[j][i] = v;
            }
        }
    }
    __device__ __forceinline__ void load(const DeltaArgs& a, int t, int lane, float (&x)[NI]) const {
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int c = lane + 32 * i;
            x[i] = c < n ? a.proj[(size_t)t * a.width + col + c] : 0.f;
        }
    }
    __device__ __forceinline__ void step(const float (&x)[NI], float (&y)[NI]) {
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            float s = 0.f;
#pragma unroll
            for (int j = 0; j < TT - 1; ++j) s = fmaf(w[j][i], win[j][i], s);
            s = fmaf(w[TT - 1][i], x[i], s);
            y[i] = silu1(s);
#pragma unroll
            for (int j = 0; j + 1 < TT - 1; ++j) win[j][i] = win[j + 1][i];
            win[TT - 2][i] = x[i];
        }
    }
};

constexpr int DP_RUN = 8;              // consecutive tokens a warp takes
constexpr int DP_WARPS = 4;

// One warp a (run of tokens, head): a key head's q and k together, or a value head.
template <int NI, int TT>
__global__ void __launch_bounds__(DP_WARPS * 32)
delta_prep_kernel(const DeltaArgs a, float* __restrict__ out) {
    chain_release();
    __shared__ float dots_s[DP_WARPS][DP_RUN][3];
    const int lane = threadIdx.x & 31, unit = blockIdx.y * DP_WARPS + (threadIdx.x >> 5);
    if (unit >= a.G + a.H) return;
    const Prepared to(a.n_tokens, a.H, a.G, a.er, a.fr);
    const int t_begin = blockIdx.x * DP_RUN, t_end = min(t_begin + DP_RUN, a.n_tokens);
    int r_now = -1;
    if (unit < a.G) {
        const int ratio = a.H / a.G;
        ConvHead<NI, TT> hq, hk;
        hq.init(a, unit * a.e, a.e, lane);
        hk.init(a, (a.G + unit) * a.e, a.e, lane);
        chain_wait();
        // the token before the run as well, if it is of the same request: its key is wanted
        const int t_first = t_begin > 0 && a.req_of_token[t_begin - 1] == a.req_of_token[t_begin]
            ? t_begin - 1 : t_begin;
        float xq[NI], xk[NI], kp[NI];
        hq.load(a, t_first, lane, xq);
        hk.load(a, t_first, lane, xk);
#pragma unroll
        for (int i = 0; i < NI; ++i) kp[i] = 0.f;
        for (int t = t_first; t < t_end; ++t) {
            const int r = a.req_of_token[t];
            if (r != r_now) {
                const float* ring = a.ring(a.state_slot[r]);
                const int i_t = t - a.cu_q[r], p = a.positions[t];
                hq.fill(a, t, i_t, p, ring, lane);
                hk.fill(a, t, i_t, p, ring, lane);
                r_now = r;
            }
            // the next token's inputs are under way while this one's are worked on
            float yq[NI], yk[NI], nq[NI], nk[NI];
            const int next = min(t + 1, t_end - 1);
            hq.load(a, next, lane, nq);
            hk.load(a, next, lane, nk);
            hq.step(xq, yq);
            hk.step(xk, yk);
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                xq[i] = nq[i];
                xk[i] = nk[i];
            }
            float sq = 0.f, sk = 0.f, sqk = 0.f, spk = 0.f, spq = 0.f;
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                if (lane + 32 * i >= a.e) yq[i] = yk[i] = 0.f;
                sq = fmaf(yq[i], yq[i], sq);
                sk = fmaf(yk[i], yk[i], sk);
                sqk = fmaf(yq[i], yk[i], sqk);
                spk = fmaf(kp[i], yk[i], spk);
                spq = fmaf(kp[i], yq[i], spq);
            }
            const float iq = 1.0f / sqrtf(warp_sum(sq) + DR_UNIT_EPS) * a.q_scale;
            const float ik = 1.0f / sqrtf(warp_sum(sk) + DR_UNIT_EPS);
            const float kq = warp_sum(sqk) * iq * ik;
            const float pk = warp_sum(spk) * ik, pq = warp_sum(spq) * iq;
            float* row = out + to.qk(unit, t);
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const int c = lane + 32 * i;
                kp[i] = yk[i] * ik;
                if (t >= t_begin && c < a.er) {
                    row[c] = yq[i] * iq;
                    row[a.er + c] = kp[i];
                }
            }
            if (t >= t_begin && lane < 3)
                dots_s[threadIdx.x >> 5][t - t_begin][lane] = lane == 0 ? kq : lane == 1 ? pk : pq;
        }
        // the scalars of the run's tokens and of the value heads that share this key head
        __syncwarp();
        for (int u = lane; u < (t_end - t_begin) * ratio; u += 32) {
            const int tt = u / ratio, head = unit * ratio + u - tt * ratio;
            const float* src = a.proj + (size_t)(t_begin + tt) * a.width;
            const float* dots = dots_s[threadIdx.x >> 5][tt];
            const float g = expf(-a.a_exp[head] * softplus1(src[a.a_col + head] + a.dt_bias[head]));
            float4* dst = reinterpret_cast<float4*>(out + to.scalars(head, t_begin + tt));
            dst[0] = make_float4(g, sigmoid1(src[a.b_col + head]), dots[0], dots[1]);
            dst[1] = make_float4(dots[2], 0.f, 0.f, 0.f);
        }
    } else {
        const int head = unit - a.G;
        ConvHead<NI, TT> hv;
        hv.init(a, 2 * a.G * a.e + head * a.f, a.f, lane);
        chain_wait();
        float x[NI];
        hv.load(a, t_begin, lane, x);
        for (int t = t_begin; t < t_end; ++t) {
            const int r = a.req_of_token[t];
            if (r != r_now) {
                hv.fill(a, t, t - a.cu_q[r], a.positions[t], a.ring(a.state_slot[r]), lane);
                r_now = r;
            }
            float y[NI], nx[NI];
            hv.load(a, min(t + 1, t_end - 1), lane, nx);
            hv.step(x, y);
#pragma unroll
            for (int i = 0; i < NI; ++i) x[i] = nx[i];
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const int c = lane + 32 * i;
                if (c < a.fr)
                    out[to.v(head, c / DR_COLS, t) + c % DR_COLS] = c < a.f ? y[i] : 0.f;
            }
        }
    }
}

constexpr int DS_COLS = DR_COLS;       // columns of S a CTA of the scan owns
constexpr int DS_TOKENS = 16;          // tokens in one of the two buffers

// R4: groups of four rows a lane keeps, er = 32 R4.  C: columns a lane keeps (a warp has 4 C): with
// two, what a lane reads of k and q serves twice.
template <int R4, int C>
__global__ void __launch_bounds__(128 / C)
delta_scan_kernel(const DeltaArgs a, const float* __restrict__ rows, float* __restrict__ out,
                  int* status) {
    using namespace mls_tma;
    constexpr int ER = 32 * R4, QK = 2 * ER;           // floats of a token's q and k
    constexpr int DS_THREADS = 128 / C;
    constexpr int V_AT = DS_TOKENS * QK, S_AT = V_AT + DS_TOKENS * DS_COLS;
    constexpr int BUF = S_AT + DS_TOKENS * DR_SCALARS;
    chain_release();
    // two buffers, and room for the rows read ahead behind the last token (not used)
    extern __shared__ __align__(128) float smem[];
    __shared__ int arrived;
    __shared__ __align__(8) uint64_t full_bars[2];
    const int r = blockIdx.z, head = blockIdx.y, col0 = blockIdx.x * DS_COLS;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, grp = lane & 7;
    const int my = warp * 4 * C + (lane >> 3);         // my columns: this one and every fourth behind it
    const Prepared from(a.n_tokens, a.H, a.G, ER, a.fr);
    const int t0 = a.cu_q[r], n = a.cu_q[r + 1] - t0;
    if (n <= 0) return;
    const int slot = a.state_slot[r];
    if (threadIdx.x == 0) {
        mbar_init((uint32_t)__cvta_generic_to_shared(&full_bars[0]), 1);
        mbar_init((uint32_t)__cvta_generic_to_shared(&full_bars[1]), 1);
        fence_barrier_init();
    }
    __syncthreads();
    chain_wait();
    auto fetch = [&](int b0) {                          // one thread: tokens b0 .. into their buffer
        const int which = (b0 / DS_TOKENS) & 1;
        const uint32_t nb = (uint32_t)min(DS_TOKENS, n - b0);
        const uint32_t bar = (uint32_t)__cvta_generic_to_shared(&full_bars[which]);
        const uint32_t dst = (uint32_t)__cvta_generic_to_shared(smem + (size_t)which * BUF);
        mbar_arrive_expect_tx(bar, nb * (uint32_t)((QK + DS_COLS + DR_SCALARS) * sizeof(float)));
        bulk_load_1d(dst, rows + from.qk(head / (a.H / a.G), t0 + b0), nb * QK * 4, bar);
        bulk_load_1d(dst + V_AT * 4, rows + from.v(head, blockIdx.x, t0 + b0), nb * DS_COLS * 4, bar);
        bulk_load_1d(dst + S_AT * 4, rows + from.scalars(head, t0 + b0), nb * DR_SCALARS * 4, bar);
    };
    if (threadIdx.x == 0) {
        fetch(0);
        if (n > DS_TOKENS) fetch(DS_TOKENS);
    }
    float* S = a.state + (size_t)slot * a.state_stride +
               ((size_t)head * a.fr + col0 + my) * ER + 4 * grp;
    f32x2 s[C][R4][2];
#pragma unroll
    for (int ci = 0; ci < C; ++ci)
#pragma unroll
        for (int i = 0; i < R4; ++i) {
            const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(S + 4 * ci * ER + 32 * i);
            s[ci][i][0] = v.x;
            s[ci][i][1] = v.y;
        }
    // the convolution's last inputs (the preparation has read the older ones)
    {
        const int keep = a.taps - 1, i0 = max(0, n - keep);
        float* ring = a.ring(slot);
        const int part = (int)(blockIdx.y * gridDim.x + blockIdx.x) * DS_THREADS + threadIdx.x;
        const int step = (int)(gridDim.x * gridDim.y) * DS_THREADS;
        for (int i = i0; i < n && keep > 0; ++i) {
            const size_t row = (size_t)(a.positions[t0 + i] % a.taps) * a.channels;
            for (int c = part; c < a.channels; c += step)
                ring[row + c] = a.proj[(size_t)(t0 + i) * a.width + a.qkv_col + c];
        }
    }
    const size_t o_row = (size_t)a.H * a.f;
    float* o_at = out + (size_t)t0 * o_row + (size_t)head * a.f + col0 + my;
    auto load_rows = [&](ulonglong2 (&v)[R4], const float* src) {
#pragma unroll
        for (int i = 0; i < R4; ++i) v[i] = *reinterpret_cast<const ulonglong2*>(src + 32 * i + 4 * grp);
    };
    auto state_dot = [&](const f32x2 (&st)[R4][2], const ulonglong2 (&v)[R4]) {   // a lane's share
        f32x2 d0 = 0ull, d1 = 0ull;
#pragma unroll
        for (int i = 0; i < R4; ++i) {
            d0 = fma2(st[i][0], v[i].x, d0);
            d1 = fma2(st[i][1], v[i].y, d1);
        }
        return sum2(add2(d0, d1));
    };
    for (int b0 = 0; b0 < n; b0 += DS_TOKENS) {
        const int nb = min(DS_TOKENS, n - b0), pass = b0 / DS_TOKENS;
        if (threadIdx.x == 0)
            arrived = mbar_wait((uint32_t)__cvta_generic_to_shared(&full_bars[pass & 1]),
                                (pass >> 1) & 1) ? 1 : 0;
        __syncthreads();
        if (!arrived) {                                 // every thread leaves at the same place
            if (threadIdx.x == 0) {                     // (once the copies under way are done, or given up)
                if (status) atomicOr(status, MLS_STATUS_TIMEOUT);
                mbar_wait((uint32_t)__cvta_generic_to_shared(&full_bars[pass & 1]), (pass >> 1) & 1);
                if (b0 + DS_TOKENS < n)
                    mbar_wait((uint32_t)__cvta_generic_to_shared(&full_bars[(pass + 1) & 1]),
                              ((pass + 1) >> 1) & 1);
            }
            return;
        }
        const float* buf = smem + (size_t)(pass & 1) * BUF;
        ulonglong2 ka[R4], qa[R4], kb[R4], qb[R4];
        load_rows(qa, buf);
        load_rows(ka, buf + ER);
        load_rows(qb, buf + QK);
        load_rows(kb, buf + QK + ER);
        float keep[C];                                  // lane grp keeps the output of one token of eight
        auto store = [&](int first, int count) {        // of the eight tokens from `first` on
            if (grp < count) {
#pragma unroll
                for (int ci = 0; ci < C; ++ci)
                    if (col0 + my + 4 * ci < a.f)
                        o_at[(size_t)(b0 + first + grp) * o_row + 4 * ci] = keep[ci];
            }
        };
        // Two tokens at a time: both tokens' products with the state before them cross the lanes
        // together, and what the first token changed of the second's follows from the products
        // of its key with the second's key and query.
        auto pair = [&](int tt) {
            const float* tok = buf + tt * QK;
            const float* sc = buf + S_AT + tt * DR_SCALARS;
            const float* v = buf + V_AT + tt * DS_COLS + my;
            float sqa[C], sqb[C], ska[C], skb[C];
#pragma unroll
            for (int ci = 0; ci < C; ++ci) {
                ska[ci] = state_dot(s[ci], ka);
                skb[ci] = state_dot(s[ci], kb);
                sqa[ci] = state_dot(s[ci], qa);
                sqb[ci] = state_dot(s[ci], qb);
            }
            const float4 ca = *reinterpret_cast<const float4*>(sc);
            const float4 cb = *reinterpret_cast<const float4*>(sc + DR_SCALARS);
            const float kqb = sc[DR_SCALARS + 4];
            load_rows(qa, tok + 2 * QK);
            load_rows(qb, tok + 3 * QK);
#pragma unroll
            for (int o = 1; o < 8; o <<= 1)
#pragma unroll
                for (int ci = 0; ci < C; ++ci) {
                    ska[ci] += __shfl_xor_sync(0xffffffffu, ska[ci], o);
                    skb[ci] += __shfl_xor_sync(0xffffffffu, skb[ci], o);
                    sqa[ci] += __shfl_xor_sync(0xffffffffu, sqa[ci], o);
                    sqb[ci] += __shfl_xor_sync(0xffffffffu, sqb[ci], o);
                }
            const float gab = ca.x * cb.x;
            const f32x2 g2 = pack2(gab, gab);
#pragma unroll
            for (int ci = 0; ci < C; ++ci) {
#pragma unroll
                for (int i = 0; i < R4; ++i) {
                    s[ci][i][0] = mul2(g2, s[ci][i][0]);
                    s[ci][i][1] = mul2(g2, s[ci][i][1]);
                }
                const float va = v[4 * ci], vb = v[DS_COLS + 4 * ci];
                const float ua = ca.y * fmaf(-ca.x, ska[ci], va);
                const float ub = cb.y * fmaf(-cb.x, fmaf(ca.x, skb[ci], cb.w * ua), vb);
                const float wa = cb.x * ua;              // the first write, decayed once
                const f32x2 a2 = pack2(wa, wa), b2 = pack2(ub, ub);
#pragma unroll
                for (int i = 0; i < R4; ++i) {
                    s[ci][i][0] = fma2(kb[i].x, b2, fma2(ka[i].x, a2, s[ci][i][0]));
                    s[ci][i][1] = fma2(kb[i].y, b2, fma2(ka[i].y, a2, s[ci][i][1]));
                }
                const float oa = fmaf(ca.x, sqa[ci], ca.z * ua);
                const float ob = fmaf(cb.x, fmaf(ca.x, sqb[ci], kqb * ua), cb.z * ub);
                if (grp == (tt & 7)) keep[ci] = oa;
                if (grp == (tt & 7) + 1) keep[ci] = ob;
            }
            load_rows(ka, tok + 2 * QK + ER);
            load_rows(kb, tok + 3 * QK + ER);
            if ((tt & 7) == 6) store(tt - 6, 8);
        };
        if (nb == DS_TOKENS) {
#pragma unroll 4
            for (int tt = 0; tt < DS_TOKENS; tt += 2) pair(tt);
        } else {
            int tt = 0;
#pragma unroll 1
            for (; tt + 1 < nb; tt += 2) pair(tt);
            if (tt < nb) {
                const float4 c = *reinterpret_cast<const float4*>(buf + S_AT + tt * DR_SCALARS);
                const f32x2 g2 = pack2(c.x, c.x);
#pragma unroll
                for (int ci = 0; ci < C; ++ci) {
                    const float sk = column_sum(state_dot(s[ci], ka)), sq = column_sum(state_dot(s[ci], qa));
                    const float u = c.y * fmaf(-c.x, sk, buf[V_AT + tt * DS_COLS + my + 4 * ci]);
                    const f32x2 u2 = pack2(u, u);
#pragma unroll
                    for (int i = 0; i < R4; ++i) {
                        s[ci][i][0] = fma2(ka[i].x, u2, mul2(g2, s[ci][i][0]));
                        s[ci][i][1] = fma2(ka[i].y, u2, mul2(g2, s[ci][i][1]));
                    }
                    if (grp == (tt & 7)) keep[ci] = fmaf(c.x, sq, c.z * u);
                }
                ++tt;
            }
            if (tt & 7) store(tt & ~7, tt & 7);
        }
        __syncthreads();                                // every read of this buffer is done
        if (threadIdx.x == 0 && b0 + 2 * DS_TOKENS < n) fetch(b0 + 2 * DS_TOKENS);
    }
#pragma unroll
    for (int ci = 0; ci < C; ++ci)
#pragma unroll
        for (int i = 0; i < R4; ++i)
            *reinterpret_cast<ulonglong2*>(S + 4 * ci * ER + 32 * i) =
                make_ulonglong2(s[ci][i][0], s[ci][i][1]);
}

constexpr int DT_THREADS = 256;        // eight warps of a (request, head)

// One token a request: convolution, unit vectors, the state's step, head norm and gate.  C:
// columns a lane keeps at a time (a pass of the block takes 32 C columns).
template <int R4, int C, typename T>
__global__ void __launch_bounds__(DT_THREADS)
delta_step_kernel(const DeltaArgs a, const float* __restrict__ norm_w, float eps,
                  T* __restrict__ out) {
    constexpr int ER = 32 * R4;
    chain_release();
    extern __shared__ __align__(128) float smem[];
    float* q_s = smem;                                  // [ER]
    float* k_s = q_s + ER;                              // [ER]
    float* v_s = k_s + ER;                              // [fr]
    float* o_s = v_s + a.fr;                            // [fr]
    float* old_s = o_s + a.fr;                          // [2 e + f]: the older taps' share
    float* now_s = old_s + 2 * a.e + a.f;               // [2 e + f]: the current token's tap
    __shared__ float sums[3];
    __shared__ float gb[2];
    const int r = blockIdx.y, head = blockIdx.x, t = a.cu_q[r];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, grp = lane & 7;
    const int ratio = a.H / a.G, kv = head / ratio;
    const int slot = a.state_slot[r], p = a.positions[t];
    float* S = a.state + (size_t)slot * a.state_stride + (size_t)head * a.fr * ER + 4 * grp;
    float* ring = a.ring(slot);
    // nothing of the state slot is written by this step's earlier kernels, so the state and the
    // convolution's older inputs are read ahead of the wait
    f32x2 s[C][R4][2];
    auto load_columns = [&](int c0) {
#pragma unroll
        for (int ci = 0; ci < C; ++ci) {
            const int col = c0 + (warp * C + ci) * 4 + (lane >> 3);
#pragma unroll
            for (int i = 0; i < R4; ++i) {
                ulonglong2 v = make_ulonglong2(0ull, 0ull);
                if (col < a.fr)
                    v = *reinterpret_cast<const ulonglong2*>(S + (size_t)col * ER + 32 * i);
                s[ci][i][0] = v.x;
                s[ci][i][1] = v.y;
            }
        }
    };
    load_columns(0);
    const int locals = 2 * a.e + a.f;
    auto channel_of = [&](int u) {                      // a local channel's place among all
        return u < a.e ? kv * a.e + u
             : u < 2 * a.e ? (a.G + kv) * a.e + (u - a.e)
                           : 2 * a.G * a.e + head * a.f + (u - 2 * a.e);
    };
    for (int u = threadIdx.x; u < locals; u += DT_THREADS) {
        const int c = channel_of(u);
        float acc = 0.f;
        for (int j = 0; j + 1 < a.taps; ++j) {
            const int back = a.taps - 1 - j;
            if (back <= p)
                acc = fmaf(load_as_float(a.conv, (size_t)c * a.taps + j, a.conv_dtype),
                           ring[(size_t)((p - back) % a.taps) * a.channels + c], acc);
        }
        old_s[u] = acc;
        now_s[u] = load_as_float(a.conv, (size_t)c * a.taps + a.taps - 1, a.conv_dtype);
    }
    for (int i = threadIdx.x; i < ER; i += DT_THREADS)
        if (i >= a.e) q_s[i] = k_s[i] = 0.f;
    for (int i = threadIdx.x; i < a.fr; i += DT_THREADS)
        if (i >= a.f) v_s[i] = 0.f;
    const float a_exp = a.a_exp[head], dt = a.dt_bias[head];
    chain_wait();
    const bool keeps_qk = head % ratio == 0;
    const size_t ring_row = (size_t)(p % a.taps) * a.channels;
    for (int u = threadIdx.x; u < locals; u += DT_THREADS) {
        const int c = channel_of(u);
        const float x = a.at(t, a.qkv_col + c);
        const float y = silu1(fmaf(now_s[u], x, old_s[u]));
        if (u < a.e) q_s[u] = y;
        else if (u < 2 * a.e) k_s[u - a.e] = y;
        else v_s[u - 2 * a.e] = y;
        if (a.taps > 1 && (keeps_qk || u >= 2 * a.e)) ring[ring_row + c] = x;
    }
    if (threadIdx.x == DT_THREADS - 1) {
        gb[0] = expf(-a_exp * softplus1(a.at(t, a.a_col + head) + dt));
        gb[1] = sigmoid1(a.at(t, a.b_col + head));
    }
    __syncthreads();
    if (warp < 3) {
        const float* x = warp == 1 ? k_s : q_s;
        const float* y = warp == 0 ? q_s : k_s;
        float v = 0.f;
#pragma unroll
        for (int i = 0; i < R4; ++i) v = fmaf(x[lane + 32 * i], y[lane + 32 * i], v);
        v = warp_sum(v);
        if (lane == 0) sums[warp] = v;
    }
    __syncthreads();
    const float iq = 1.0f / sqrtf(sums[0] + DR_UNIT_EPS) * a.q_scale;
    const float ik = 1.0f / sqrtf(sums[1] + DR_UNIT_EPS);
    const float kq = sums[2] * iq * ik, g = gb[0], beta = gb[1];
    const f32x2 g2 = pack2(g, g);
    for (int c0 = 0; c0 < a.fr; c0 += 32 * C) {
        if (c0 > 0) load_columns(c0);
        f32x2 dk[C], dq[C];
#pragma unroll
        for (int ci = 0; ci < C; ++ci) dk[ci] = dq[ci] = 0ull;
#pragma unroll
        for (int i = 0; i < R4; ++i) {
            const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(k_s + 32 * i + 4 * grp);
            const ulonglong2 q = *reinterpret_cast<const ulonglong2*>(q_s + 32 * i + 4 * grp);
#pragma unroll
            for (int ci = 0; ci < C; ++ci) {
                dk[ci] = fma2(s[ci][i][0], k.x, dk[ci]);
                dq[ci] = fma2(s[ci][i][0], q.x, dq[ci]);
                dk[ci] = fma2(s[ci][i][1], k.y, dk[ci]);
                dq[ci] = fma2(s[ci][i][1], q.y, dq[ci]);
            }
        }
        f32x2 u2[C];
#pragma unroll
        for (int ci = 0; ci < C; ++ci) {
            const int col = c0 + (warp * C + ci) * 4 + (lane >> 3);
            const float sk = column_sum(sum2(dk[ci])) * ik, sq = column_sum(sum2(dq[ci])) * iq;
            const float u = col < a.fr ? beta * fmaf(-g, sk, v_s[col]) : 0.f;
            u2[ci] = pack2(u * ik, u * ik);
            if (grp == 0 && col < a.fr) o_s[col] = fmaf(g, sq, kq * u);
        }
#pragma unroll
        for (int i = 0; i < R4; ++i) {
            const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(k_s + 32 * i + 4 * grp);
#pragma unroll
            for (int ci = 0; ci < C; ++ci) {
                const int col = c0 + (warp * C + ci) * 4 + (lane >> 3);
                if (col < a.fr)
                    *reinterpret_cast<ulonglong2*>(S + (size_t)col * ER + 32 * i) =
                        make_ulonglong2(fma2(k.x, u2[ci], mul2(g2, s[ci][i][0])),
                                        fma2(k.y, u2[ci], mul2(g2, s[ci][i][1])));
            }
        }
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = lane; c < a.f; c += 32) ss = fmaf(o_s[c], o_s[c], ss);     // every warp for itself
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)a.f + eps);
    for (int c = threadIdx.x; c < a.f; c += DT_THREADS) {
        const float z = a.at(t, a.g_col + head * a.f + c);
        Elem<T>::store(out + (size_t)t * a.H * a.f + head * a.f + c,
                       o_s[c] * inv * norm_w[c] * silu1(z));
    }
}

DeltaArgs make_args(const float* proj, int n_parts, long long part_stride, int width, int qkv_col,
                    int a_col, int b_col, int g_col, const void* conv, int conv_dtype, int taps,
                    const float* a_exp, const float* dt_bias, const int* state_slot,
                    const int* cu_q, const int* req_of_token, const int* positions, float* state,
                    long long state_stride, int n_tokens, int n_requests, int H, int G, int e,
                    int f) {
    DeltaArgs a;
    a.proj = proj; a.n_parts = n_parts; a.part_stride = part_stride; a.width = width;
    a.qkv_col = qkv_col; a.a_col = a_col; a.b_col = b_col; a.g_col = g_col; a.conv = conv;
    a.conv_dtype = conv_dtype; a.taps = taps; a.channels = 2 * G * e + H * f; a.a_exp = a_exp;
    a.dt_bias = dt_bias; a.state_slot = state_slot; a.cu_q = cu_q; a.req_of_token = req_of_token;
    a.positions = positions; a.state = state; a.state_stride = state_stride;
    a.n_tokens = n_tokens; a.n_requests = n_requests; a.H = H; a.G = G; a.e = e; a.f = f;
    a.er = (e + 31) / 32 * 32;
    a.fr = (f + 15) / 16 * 16;
    a.ring_at = (long long)H * a.fr * a.er;
    a.q_scale = 1.0f / sqrtf((float)e);
    return a;
}
bool sizes_ok(const DeltaArgs& a) {
    return a.H > 0 && a.G > 0 && a.H % a.G == 0 && a.e > 0 && a.e <= 256 && a.f > 0 && a.taps >= 1 &&
           a.n_parts >= 1 && a.state_stride % 4 == 0 &&
           a.state_stride >= a.ring_at + (long long)a.taps * a.channels;
}

template <int NI>
int launch_prep(const DeltaArgs& a, float* out, cudaStream_t stream) {
    const dim3 grid((a.n_tokens + DP_RUN - 1) / DP_RUN, (a.G + a.H + DP_WARPS - 1) / DP_WARPS);
    if (a.taps <= 4) MLS_LAUNCH((delta_prep_kernel<NI, 4>), grid, dim3(DP_WARPS * 32), 0, stream, a, out);
    else if (a.taps <= 8) MLS_LAUNCH((delta_prep_kernel<NI, 8>), grid, dim3(DP_WARPS * 32), 0, stream, a, out);
    else MLS_LAUNCH((delta_prep_kernel<NI, 16>), grid, dim3(DP_WARPS * 32), 0, stream, a, out);
    return launch_status();
}
template <int R4, int C>
int launch_scan(const DeltaArgs& a, const float* rows, float* out, int* status,
                cudaStream_t stream) {
    constexpr size_t qk = 2 * 32 * R4;
    const size_t smem = (2 * DS_TOKENS * (qk + DS_COLS + DR_SCALARS) + 4 * qk) * sizeof(float);
    if (smem > 40 * 1024) {                             // (static shared memory comes on top)
        const int rc = (int)cudaFuncSetAttribute(
            delta_scan_kernel<R4, C>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (rc) return rc;
    }
    MLS_LAUNCH((delta_scan_kernel<R4, C>), dim3(a.fr / DS_COLS, a.H, a.n_requests), dim3(128 / C),
               smem, stream, a, rows, out, status);
    return launch_status();
}
template <int R4, int C>
int launch_step(const DeltaArgs& a, const float* norm_w, float eps, void* out, int dtype,
                cudaStream_t stream) {
    const size_t smem = ((size_t)2 * 32 * R4 + 2 * a.fr + 2 * (2 * a.e + a.f)) * sizeof(float);
    if (smem > 200 * 1024) return MLS_ERR_UNSUPPORTED;
    if (dtype == MLS_BF16) {
        auto kernel = delta_step_kernel<R4, C, __nv_bfloat16>;
        if (smem > 40 * 1024) {
            const int rc = (int)cudaFuncSetAttribute(
                kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            if (rc) return rc;
        }
        MLS_LAUNCH(kernel, dim3(a.H, a.n_requests), dim3(DT_THREADS), smem, stream, a, norm_w, eps,
                   (__nv_bfloat16*)out);
    } else {
        auto kernel = delta_step_kernel<R4, C, float>;
        if (smem > 40 * 1024) {
            const int rc = (int)cudaFuncSetAttribute(
                kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            if (rc) return rc;
        }
        MLS_LAUNCH(kernel, dim3(a.H, a.n_requests), dim3(DT_THREADS), smem, stream, a, norm_w, eps,
                   (float*)out);
    }
    return launch_status();
}
}  // namespace

// Floats of a token's share of what the scan reads, and of a request's state.
MLS_API int mls_delta_row_floats(int H, int G, int e, int f) {
    return prepared_floats(H, G, (e + 31) / 32 * 32, (f + 15) / 16 * 16);
}
MLS_API long long mls_delta_state_floats(int H, int G, int e, int f, int taps) {
    const long long s = (long long)H * ((f + 15) / 16 * 16) * ((e + 31) / 32 * 32) +
                        (long long)taps * (2LL * G * e + (long long)H * f);
    return (s + 3) / 4 * 4;
}

// Preparation and scan of the tokens of a step (rows: scratch, [T, mls_delta_row_floats]);
// out [T, H f] float32.
MLS_API int mls_delta_prep(const float* proj, int width, int qkv_col, int a_col, int b_col,
                           const void* conv, int conv_dtype, int taps, const float* a_exp,
                           const float* dt_bias, const int* state_slot, const int* cu_q,
                           const int* req_of_token, const int* positions, float* state,
                           long long state_stride, int n_tokens, int n_requests, int H, int G,
                           int e, int f, float* rows, cudaStream_t stream) {
    if (n_tokens <= 0 || n_requests <= 0) return 0;
    const DeltaArgs a = make_args(proj, 1, 0, width, qkv_col, a_col, b_col, 0, conv, conv_dtype, taps,
                                  a_exp, dt_bias, state_slot, cu_q, req_of_token, positions, state,
                                  state_stride, n_tokens, n_requests, H, G, e, f);
    if (!sizes_ok(a) || taps > 16 || a.fr > 256) return MLS_ERR_UNSUPPORTED;
    const int ni = (max(a.er, a.fr) + 31) / 32;
    if (ni <= 1) return launch_prep<1>(a, rows, stream);
    if (ni <= 2) return launch_prep<2>(a, rows, stream);
    if (ni <= 4) return launch_prep<4>(a, rows, stream);
    return launch_prep<8>(a, rows, stream);
}

MLS_API int mls_delta_scan(const float* rows, const float* proj, int width, int qkv_col, int taps,
                           const int* state_slot, const int* cu_q, const int* positions,
                           float* state, long long state_stride, int n_tokens, int n_requests,
                           int H, int G, int e, int f, float* out, int* status,
                           cudaStream_t stream) {
    if (n_tokens <= 0 || n_requests <= 0) return 0;
    const DeltaArgs a = make_args(proj, 1, 0, width, qkv_col, 0, 0, 0, nullptr, 0, taps, nullptr, nullptr,
                                  state_slot, cu_q, nullptr, positions, state, state_stride,
                                  n_tokens, n_requests, H, G, e, f);
    if (!sizes_ok(a) || n_requests > 65535 || H > 65535) return MLS_ERR_UNSUPPORTED;
    // one column a lane while every CTA has an SM to itself (more warps to hide the chain of
    // products and sums), two beyond that (half the reads of k and q); the bits are the same
    const bool one = (long long)(a.fr / DS_COLS) * H * n_requests <= sm_count();
#define DS_GO(R, C) return launch_scan<R, C>(a, rows, out, status, stream)
    switch (a.er / 32) {
        case 1: if (one) DS_GO(1, 1); DS_GO(1, 2);
        case 2: if (one) DS_GO(2, 1); DS_GO(2, 2);
        case 3: if (one) DS_GO(3, 1); DS_GO(3, 2);
        case 4: if (one) DS_GO(4, 1); DS_GO(4, 2);
        case 5: DS_GO(5, 1);
        case 6: DS_GO(6, 1);
        case 7: DS_GO(7, 1);
        default: DS_GO(8, 1);
    }
#undef DS_GO
}

// A step of one token a request, to the gated and normed heads: out [T, H f] in `dtype`.
MLS_API int mls_delta_step(const float* proj, int n_parts, long long part_stride, int width,
                           int qkv_col, int a_col, int b_col, int g_col, const void* conv,
                           int conv_dtype, int taps, const float* a_exp, const float* dt_bias,
                           const float* norm_w, float eps, const int* state_slot, const int* cu_q,
                           const int* positions, float* state, long long state_stride,
                           int n_requests, int H, int G, int e, int f, void* out, int dtype,
                           cudaStream_t stream) {
    if (n_requests <= 0) return 0;
    const DeltaArgs a = make_args(proj, n_parts, part_stride, width, qkv_col, a_col, b_col, g_col, conv,
                                  conv_dtype, taps, a_exp, dt_bias, state_slot, cu_q, nullptr,
                                  positions, state, state_stride, n_requests, n_requests, H, G, e, f);
    if (!sizes_ok(a) || n_requests > 65535) return MLS_ERR_UNSUPPORTED;
    switch (a.er / 32) {
        case 1: return launch_step<1, 8>(a, norm_w, eps, out, dtype, stream);
        case 2: return launch_step<2, 8>(a, norm_w, eps, out, dtype, stream);
        case 3: return launch_step<3, 4>(a, norm_w, eps, out, dtype, stream);
        case 4: return launch_step<4, 4>(a, norm_w, eps, out, dtype, stream);
        case 5: return launch_step<5, 2>(a, norm_w, eps, out, dtype, stream);
        case 6: return launch_step<6, 2>(a, norm_w, eps, out, dtype, stream);
        case 7: return launch_step<7, 2>(a, norm_w, eps, out, dtype, stream);
        default: return launch_step<8, 2>(a, norm_w, eps, out, dtype, stream);
    }
}
