// Gated linear recurrence over channels (one float per request and channel instead of a matrix per head):
//
//   p = (Wx h) + bx          u_t = sum_m c[ch, m] p_(t - K + 1 + m) + cb       causal, per channel, p = 0 before the sequence's start
//   per part b of the channels (equal parts):  r = sg(Ra_b u_b + ra_b),  i = sg(Ri_b u_b + ri_b)
//   l = r * nsp (nsp = -8 softplus(lam) per channel);  S_t = e^l S_(t-1) + sqrt(1 - e^(2 l)) i u;   out = T( S * gelu_tanh((Wy h) + by) )
//
// A request's state row holds S [W] and behind it, for K > 1 taps, a ring of the last K inputs p [K, W]: the input at position
// q lies in row q mod K.  A ring of K rows (one more than the convolution looks back) lets the kernel for decoded tokens write its
// input while other blocks still read the others; inputs before position 0 are zeros by their position, so a slot needs no
// clearing for them.  Everything that enters the recurrence is float; u is rounded once to the activations' type T.
//
//   lru_conv   : u of every token of the step
//   (the two gate products of every part are one batched library product into z [parts, T, 2 * part], float)
//   lru_chunk  : per chunk of a request's tokens and channel: a = e^l and the weighted input, which replace the two products in z,
//                and what the chunk does to a state: the product of its a and the state it leaves from zero.  A request's first
//                chunk starts from the request's state instead and leaves that state beside the one it ends with.
//   lru_finish : per chunk and channel: the state in front of the chunk from the summaries of the chunks before it, then the
//                tokens one after the other; the gate; a request's last chunk leaves the new state and the ring.  Where no
//                request has more than one chunk it works from the gate products directly and lru_chunk is not launched.
//   lru_step   : a step of decoded tokens (one per request): all of it in one kernel.  A block owns a few channels of one part and up
//                to eight requests: the part's convolutions into shared memory, the two rows of gate weights of a channel read once
//                for all its requests, the recurrence, the gate, the ring.
#include "common.cuh"

namespace cvb {

constexpr int kLruThreads = 128;

__device__ __forceinline__ float lru_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float lru_gelu(float z) { return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))); }

struct LruShape {
    int W, part, taps, stride;          // channels, channels per part, taps, elements per row of the packed projection
    int y_off, x_off;                   // columns of the two projections
    int64_t state_floats;
    int num_slots;
};

// u of channel c for the token at packed row t: `local` tokens of its portion lie before it, it sits at position pos.
template <typename T>
__device__ __forceinline__ float lru_conv_of(const T* __restrict__ packed, const float* __restrict__ bias_x, const float* __restrict__ conv_w,
                                             const float* __restrict__ conv_b, const float* __restrict__ ring, const LruShape& sh, int64_t t,
                                             int local, int pos, int c) {
    float acc = 0.f;
    const float b = bias_x[c];
    for (int m = 0; m < sh.taps; ++m) {
        const int back = sh.taps - 1 - m;
        float x = 0.f;
        if (local >= back) x = to_float(packed[(t - back) * sh.stride + sh.x_off + c]) + b;
        else if (pos >= back) x = ring[static_cast<int64_t>((pos - back) % sh.taps) * sh.W + c];
        acc = fmaf(conv_w[static_cast<int64_t>(m) * sh.W + c], x, acc);
    }
    return acc + conv_b[c];
}

template <typename T>
__global__ void __launch_bounds__(kLruThreads)
lru_conv_kernel(T* __restrict__ u, const T* __restrict__ packed, const float* __restrict__ bias_x, const float* __restrict__ conv_w,
                const float* __restrict__ conv_b, const float* __restrict__ state, const int* __restrict__ seq_of_token,
                const int* __restrict__ cu_seqlens, const int* __restrict__ state_slots, const int* __restrict__ positions, LruShape sh,
                int* __restrict__ err) {
    pdl_trigger();
    pdl_wait();
    const int64_t t = blockIdx.x;
    const int s = seq_of_token[t];
    const int slot = state_slots[s];
    if (slot < 0 || slot >= sh.num_slots) {
        if (threadIdx.x == 0) atomicExch(err, 2);
        return;
    }
    const int local = static_cast<int>(t) - cu_seqlens[s], pos = positions[t];
    const float* ring = state + static_cast<int64_t>(slot) * sh.state_floats + sh.W;
    for (int c = blockIdx.y * kLruThreads + threadIdx.x; c < sh.W; c += gridDim.y * kLruThreads)
        u[t * sh.W + c] = from_float<T>(lru_conv_of(packed, bias_x, conv_w, conv_b, ring, sh, t, local, pos, c));
}

// The same by vectors: a thread owns the channels of 16 bytes over `run` neighbouring tokens of the flattened batch and slides a
// window of K rows along; a token whose window reaches back before its portion takes the general form.
template <typename T> struct LruVec;
template <> struct LruVec<float> {
    static constexpr int N = 4;
    static __device__ __forceinline__ void load(float (&f)[4], const float* p) { const float4 v = *reinterpret_cast<const float4*>(p); f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w; }
    static __device__ __forceinline__ void store(float* p, const float (&f)[4]) { *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); }
};
template <> struct LruVec<__nv_bfloat16> {
    static constexpr int N = 8;
    static __device__ __forceinline__ void load(float (&f)[8], const __nv_bfloat16* p) {
        const uint4 raw = *reinterpret_cast<const uint4*>(p);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) { const float2 v = __bfloat1622float2(h[i]); f[2 * i] = v.x; f[2 * i + 1] = v.y; }
    }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&f)[8]) {
        uint4 raw;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
        *reinterpret_cast<uint4*>(p) = raw;
    }
};

template <typename T, int K>
__global__ void __launch_bounds__(kLruThreads)
lru_conv_vec_kernel(T* __restrict__ u, const T* __restrict__ packed, const float* __restrict__ bias_x, const float* __restrict__ conv_w,
                    const float* __restrict__ conv_b, const float* __restrict__ state, const int* __restrict__ seq_of_token,
                    const int* __restrict__ cu_seqlens, const int* __restrict__ state_slots, const int* __restrict__ positions, int n_tokens,
                    int run, LruShape sh, int* __restrict__ err) {
    pdl_trigger();
    pdl_wait();
    constexpr int N = LruVec<T>::N;
    const int c = (blockIdx.y * kLruThreads + threadIdx.x) * N;
    if (c >= sh.W) return;
    const int t0 = blockIdx.x * run, t1 = min(t0 + run, n_tokens);
    float w[K][N], b[N], cb[N], x[K][N];
#pragma unroll
    for (int e = 0; e < N; ++e) { b[e] = bias_x[c + e]; cb[e] = conv_b[c + e]; }
#pragma unroll
    for (int m = 0; m < K; ++m)
#pragma unroll
        for (int e = 0; e < N; ++e) w[m][e] = conv_w[static_cast<int64_t>(m) * sh.W + c + e];
    const T* base = packed + sh.x_off + c;
#pragma unroll
    for (int m = 1; m < K; ++m) {                       // rows t0 - K + 1 .. t0 - 1; the loop shifts them into place
        const int t = t0 - K + m;
        LruVec<T>::load(x[m], base + static_cast<int64_t>(max(t, 0)) * sh.stride);
#pragma unroll
        for (int e = 0; e < N; ++e) x[m][e] += b[e];
    }
    for (int t = t0; t < t1; ++t) {
#pragma unroll
        for (int m = 0; m + 1 < K; ++m)
#pragma unroll
            for (int e = 0; e < N; ++e) x[m][e] = x[m + 1][e];
        LruVec<T>::load(x[K - 1], base + static_cast<int64_t>(t) * sh.stride);
#pragma unroll
        for (int e = 0; e < N; ++e) x[K - 1][e] += b[e];
        const int s = seq_of_token[t], local = t - cu_seqlens[s];
        float y[N];
        if (local >= K - 1) {
#pragma unroll
            for (int e = 0; e < N; ++e) {
                float acc = 0.f;
#pragma unroll
                for (int m = 0; m < K; ++m) acc = fmaf(w[m][e], x[m][e], acc);
                y[e] = acc + cb[e];
            }
        } else {
            const int slot = state_slots[s];
            if (slot < 0 || slot >= sh.num_slots) {
                atomicExch(err, 2);
                continue;
            }
            const float* ring = state + static_cast<int64_t>(slot) * sh.state_floats + sh.W;
#pragma unroll
            for (int e = 0; e < N; ++e) y[e] = lru_conv_of(packed, bias_x, conv_w, conv_b, ring, sh, t, local, positions[t], c + e);
        }
        LruVec<T>::store(u + static_cast<int64_t>(t) * sh.W + c, y);
    }
}

// Which chunk of which request block x works on: chunk k of request s holds its tokens k * len .. (at most len of them).
__device__ __forceinline__ bool lru_locate(const int* __restrict__ cu_seqlens, int S, int len, int x, int& s_out, int& k, int& first_chunk) {
    int base = 0;
    for (int s = 0; s < S; ++s) {
        const int n = cu_seqlens[s + 1] - cu_seqlens[s];
        const int chunks = (n + len - 1) / len;
        if (x < base + chunks) { s_out = s; k = x - base; first_chunk = base; return true; }
        base += chunks;
    }
    return false;
}

// 1 - e^y for y <= 0: by its series where the difference would cancel
__device__ __forceinline__ float one_minus_exp(float y) {
    const float series = y * (1.f + y * (1.f / 2.f) * (1.f + y * (1.f / 3.f) * (1.f + y * (1.f / 4.f) * (1.f + y * (1.f / 5.f) * (1.f + y * (1.f / 6.f) * (1.f + y * (1.f / 7.f)))))));
    return y > -0.5f ? -series : 1.f - __expf(y);
}

// The decay and the weighted input from the two gate products.  With bf16 activations through the hardware's exponential and
// division; in the 32-bit path through the library's functions.
template <typename T>
__device__ __forceinline__ void lru_gate(float zr, float zi, float br, float bi, float nsp, float u, float& a, float& in) {
    if constexpr (sizeof(T) == 2) {
        const float l = __fdividef(nsp, 1.f + __expf(-(zr + br)));
        a = __expf(l);
        in = __fsqrt_rn(fmaxf(one_minus_exp(2.f * l), 0.f)) * __fdividef(u, 1.f + __expf(-(zi + bi)));
    } else {
        const float l = lru_sigmoid(zr + br) * nsp;
        a = expf(l);
        in = sqrtf(fmaxf(-expm1f(2.f * l), 0.f)) * lru_sigmoid(zi + bi) * u;
    }
}

// gelu_tanh: z / 2 (1 + tanh(s)) = z sigmoid(2 s)
template <typename T>
__device__ __forceinline__ float lru_gelu_of(float z) {
    if constexpr (sizeof(T) == 2) return __fdividef(z, 1.f + __expf(-2.f * 0.7978845608028654f * (z + 0.044715f * z * z * z)));
    else return lru_gelu(z);
}

template <typename T>
__global__ void __launch_bounds__(kLruThreads)
lru_chunk_kernel(float* __restrict__ z, const T* __restrict__ u, const float* __restrict__ br, const float* __restrict__ bi,
                 const float* __restrict__ nsp, const float* __restrict__ state, float* __restrict__ summary,
                 const int* __restrict__ cu_seqlens, const int* __restrict__ state_slots, int S, int n_tokens, int len, LruShape sh,
                 int* __restrict__ err) {
    pdl_trigger();
    pdl_wait();
    int s, k, first_chunk;
    if (!lru_locate(cu_seqlens, S, len, blockIdx.x, s, k, first_chunk)) return;
    const int c = blockIdx.y * kLruThreads + threadIdx.x;
    if (c >= sh.W) return;
    const int slot = state_slots[s];
    if (slot < 0 || slot >= sh.num_slots) {
        if (threadIdx.x == 0) atomicExch(err, 2);
        return;
    }
    const int t0 = cu_seqlens[s] + k * len, n = min(len, cu_seqlens[s + 1] - t0);
    const int b = c / sh.part, o = c - b * sh.part;
    float* zp = z + (static_cast<int64_t>(b) * n_tokens + t0) * 2 * sh.part + o;
    const T* up = u + static_cast<int64_t>(t0) * sh.W + c;
    const float rb = br[c], ib = bi[c], ns = nsp[c];
    float A = 1.f, B = 0.f;
    if (k == 0) { B = state[static_cast<int64_t>(slot) * sh.state_floats + c]; }
    const float start = B;
#pragma unroll 8
    for (int i = 0; i < n; ++i) {
        float a, in;
        lru_gate<T>(zp[static_cast<int64_t>(i) * 2 * sh.part], zp[static_cast<int64_t>(i) * 2 * sh.part + sh.part], rb, ib, ns,
                 to_float(up[static_cast<int64_t>(i) * sh.W]), a, in);
        zp[static_cast<int64_t>(i) * 2 * sh.part] = a;
        zp[static_cast<int64_t>(i) * 2 * sh.part + sh.part] = in;
        A *= a;
        B = fmaf(a, B, in);
    }
    float* out = summary + static_cast<int64_t>(blockIdx.x) * 2 * sh.W + c;
    out[0] = k == 0 ? start : A;
    out[sh.W] = B;
}

template <typename T, bool GATED>
__global__ void __launch_bounds__(kLruThreads)
lru_finish_kernel(T* __restrict__ out, const float* __restrict__ z, const T* __restrict__ u, const T* __restrict__ packed,
                  const float* __restrict__ bias_y, const float* __restrict__ bias_x, const float* __restrict__ br,
                  const float* __restrict__ bi, const float* __restrict__ nsp, float* __restrict__ state, const float* __restrict__ summary,
                  const int* __restrict__ cu_seqlens, const int* __restrict__ state_slots, const int* __restrict__ positions, int S,
                  int n_tokens, int len, LruShape sh, int* __restrict__ err) {
    pdl_trigger();
    pdl_wait();
    int s, k, first_chunk;
    if (!lru_locate(cu_seqlens, S, len, blockIdx.x, s, k, first_chunk)) return;
    const int c = blockIdx.y * kLruThreads + threadIdx.x;
    if (c >= sh.W) return;
    const int slot = state_slots[s];
    if (slot < 0 || slot >= sh.num_slots) {
        if (threadIdx.x == 0) atomicExch(err, 2);
        return;
    }
    const int begin = cu_seqlens[s], end = cu_seqlens[s + 1];
    const int t0 = begin + k * len, n = min(len, end - t0);
    const int b = c / sh.part, o = c - b * sh.part;
    const float* zp = z + (static_cast<int64_t>(b) * n_tokens + t0) * 2 * sh.part + o;
    const T* up = u + static_cast<int64_t>(t0) * sh.W + c;
    const T* yp = packed + static_cast<int64_t>(t0) * sh.stride + sh.y_off + c;
    T* op = out + static_cast<int64_t>(t0) * sh.W + c;
    float* row = state + static_cast<int64_t>(slot) * sh.state_floats;
    float st;
    if (GATED) {
        st = row[c];
    } else {
        const float* sm = summary + static_cast<int64_t>(first_chunk) * 2 * sh.W + c;
        if (k == 0) {
            st = sm[0];
        } else {
            st = sm[sh.W];
#pragma unroll 4
            for (int j = 1; j < k; ++j) st = fmaf(sm[static_cast<int64_t>(j) * 2 * sh.W], st, sm[static_cast<int64_t>(j) * 2 * sh.W + sh.W]);
        }
    }
    const float rb = GATED ? br[c] : 0.f, ib = GATED ? bi[c] : 0.f, ns = GATED ? nsp[c] : 0.f, yb = bias_y[c];
    constexpr int kAhead = 8;                           // tokens whose rows are asked for together
    for (int i0 = 0; i0 < n; i0 += kAhead) {
        float a[kAhead], in[kAhead], y[kAhead], uu[kAhead];
#pragma unroll
        for (int e = 0; e < kAhead; ++e) {
            const int i = min(i0 + e, n - 1);
            a[e] = zp[static_cast<int64_t>(i) * 2 * sh.part];
            in[e] = zp[static_cast<int64_t>(i) * 2 * sh.part + sh.part];
            y[e] = to_float(yp[static_cast<int64_t>(i) * sh.stride]);
            if (GATED) uu[e] = to_float(up[static_cast<int64_t>(i) * sh.W]);
        }
#pragma unroll
        for (int e = 0; e < kAhead; ++e) {
            if (i0 + e >= n) break;
            if (GATED) lru_gate<T>(a[e], in[e], rb, ib, ns, uu[e], a[e], in[e]);
            st = fmaf(a[e], st, in[e]);
            op[static_cast<int64_t>(i0 + e) * sh.W] = from_float<T>(st * lru_gelu_of<T>(y[e] + yb));
        }
    }
    if (t0 + n == end) {
        row[c] = st;
        if (sh.taps > 1) {
            const float xb = bias_x[c];
            for (int t = max(begin, end - sh.taps); t < end; ++t)
                row[sh.W + static_cast<int64_t>(positions[t] % sh.taps) * sh.W + c] = to_float(packed[static_cast<int64_t>(t) * sh.stride + sh.x_off + c]) + xb;
        }
    }
}

constexpr int kStepThreads = 256;
constexpr int kStepTokens = 8;          // requests per block
constexpr int kStepWarps = kStepThreads / 32;

__device__ __forceinline__ void fma8(const __nv_bfloat16* w, float (&f)[8]) {
    const uint4 raw = *reinterpret_cast<const uint4*>(w);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) { const float2 v = __bfloat1622float2(h[i]); f[2 * i] = v.x; f[2 * i + 1] = v.y; }
}
__device__ __forceinline__ void fma8(const float* w, float (&f)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(w), b = *reinterpret_cast<const float4*>(w + 4);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}

// gates [parts, 2 * part, part]: the rows of Ra over the rows of Ri
// NT requests a block; K > 0: that many taps, known to the compiler
template <typename T, int NT, int K>
__global__ void __launch_bounds__(kStepThreads)
lru_step_kernel(T* __restrict__ out, const T* __restrict__ packed, const float* __restrict__ bias_y, const float* __restrict__ bias_x,
                const float* __restrict__ conv_w, const float* __restrict__ conv_b, const T* __restrict__ gates, const float* __restrict__ br,
                const float* __restrict__ bi, const float* __restrict__ nsp, float* __restrict__ state, const int* __restrict__ cu_seqlens,
                const int* __restrict__ state_slots, const int* __restrict__ positions, int S, LruShape sh, int vec, int per_warp, int* __restrict__ err) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) float us[];         // [NT][ld]
    const int chans = kStepWarps * per_warp;            // channels of the block: a warp takes every eighth of them
    const int per_part = (sh.part + chans - 1) / chans;
    const int b = blockIdx.x / per_part, o0 = (blockIdx.x - b * per_part) * chans, o1 = min(o0 + chans, sh.part);
    const int s0 = blockIdx.y * NT, nt = min(NT, S - s0);
    const int ld = (sh.part + 7) / 8 * 8;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const T* rows_r = gates + static_cast<int64_t>(b) * 2 * sh.part * sh.part;
    const T* rows_i = rows_r + static_cast<int64_t>(sh.part) * sh.part;
    float fr[8], fi[8];                                 // a channel's first 256 gate weights are on their way before they are needed
    auto ahead = [&](int o) {
        if (vec && lane * 8 < sh.part && o < o1) {
            fma8(rows_r + static_cast<int64_t>(o) * sh.part + lane * 8, fr);
            fma8(rows_i + static_cast<int64_t>(o) * sh.part + lane * 8, fi);
        }
    };
    ahead(o0 + warp);
    __shared__ int s_slot[NT], s_tok[NT], s_pos[NT];
    if (threadIdx.x < NT) {
        const int k = threadIdx.x;
        const int t = k < nt ? cu_seqlens[s0 + k] : 0;
        int slot = k < nt ? state_slots[s0 + k] : -1;
        if (slot >= sh.num_slots || (slot < 0 && k < nt)) { atomicExch(err, 2); slot = -1; }
        s_slot[k] = slot; s_tok[k] = t; s_pos[k] = positions[t];
    }
    __syncthreads();
    for (int ch = threadIdx.x; ch < sh.part; ch += kStepThreads) {
        const int c = b * sh.part + ch;
        if constexpr (K > 0) {
            float cw[K];
#pragma unroll
            for (int m = 0; m < K; ++m) cw[m] = conv_w[static_cast<int64_t>(m) * sh.W + c];
            const float xb = bias_x[c], cb = conv_b[c];
            float x[NT][K];
#pragma unroll
            for (int k = 0; k < NT; ++k) {
                const bool live = s_slot[k] >= 0;
                const float* ring = state + static_cast<int64_t>(live ? s_slot[k] : 0) * sh.state_floats + sh.W + c;
#pragma unroll
                for (int m = 0; m < K; ++m) {
                    const int back = K - 1 - m, pos = s_pos[k];
                    if (back == 0) x[k][m] = live ? to_float(packed[static_cast<int64_t>(s_tok[k]) * sh.stride + sh.x_off + c]) + xb : 0.f;
                    else x[k][m] = (live && pos >= back) ? ring[static_cast<int64_t>((pos - back) % K) * sh.W] : 0.f;
                }
            }
#pragma unroll
            for (int k = 0; k < NT; ++k) {
                float acc = 0.f;
#pragma unroll
                for (int m = 0; m < K; ++m) acc = fmaf(cw[m], x[k][m], acc);
                us[k * ld + ch] = rnd<T>(acc + cb);
            }
        } else {
            for (int k = 0; k < NT; ++k)
                us[k * ld + ch] = s_slot[k] < 0 ? 0.f
                    : rnd<T>(lru_conv_of(packed, bias_x, conv_w, conv_b, state + static_cast<int64_t>(s_slot[k]) * sh.state_floats + sh.W, sh,
                                         s_tok[k], 0, s_pos[k], c));
        }
    }
    __syncthreads();
    for (int o = o0 + warp; o < o1; o += kStepWarps) {
        const T* wr = rows_r + static_cast<int64_t>(o) * sh.part;
        const T* wi = rows_i + static_cast<int64_t>(o) * sh.part;
        // what lane k needs of request k at the end, asked for before the products
        const int c = b * sh.part + o;
        const bool mine = lane < nt && s_slot[lane < NT ? lane : 0] >= 0;
        const int t = mine ? s_tok[lane] : 0;
        float* row = state + static_cast<int64_t>(mine ? s_slot[lane] : 0) * sh.state_floats;
        float s_old = 0.f, rb = 0.f, ib = 0.f, ns = 0.f, yv = 0.f, xv = 0.f;
        if (mine) {
            s_old = row[c]; rb = br[c]; ib = bi[c]; ns = nsp[c];
            yv = to_float(packed[static_cast<int64_t>(t) * sh.stride + sh.y_off + c]) + bias_y[c];
            xv = to_float(packed[static_cast<int64_t>(t) * sh.stride + sh.x_off + c]) + bias_x[c];
        }
        float zr[NT], zi[NT];
#pragma unroll
        for (int k = 0; k < NT; ++k) zr[k] = zi[k] = 0.f;
        if (vec) {
            for (int e = lane * 8; e < sh.part; e += 256) {
                if (e >= 256) { fma8(wr + e, fr); fma8(wi + e, fi); }
#pragma unroll
                for (int k = 0; k < NT; ++k) {
                    const float4 x0 = *reinterpret_cast<const float4*>(us + k * ld + e), x1 = *reinterpret_cast<const float4*>(us + k * ld + e + 4);
                    const float x[8] = {x0.x, x0.y, x0.z, x0.w, x1.x, x1.y, x1.z, x1.w};
#pragma unroll
                    for (int j = 0; j < 8; ++j) { zr[k] = fmaf(x[j], fr[j], zr[k]); zi[k] = fmaf(x[j], fi[j], zi[k]); }
                }
            }
        } else {
            for (int e = lane; e < sh.part; e += 32) {
                const float fr = to_float(wr[e]), fi = to_float(wi[e]);
#pragma unroll
                for (int k = 0; k < NT; ++k) { const float x = us[k * ld + e]; zr[k] = fmaf(x, fr, zr[k]); zi[k] = fmaf(x, fi, zi[k]); }
            }
        }
        ahead(o + kStepWarps);
        // the 2 NT sums over the warp by a transposing butterfly: lane l ends with the sum of value l / (32 / (2 NT)), of which lane k
        // fetches request k's two
        float r[2 * NT];
#pragma unroll
        for (int k = 0; k < NT; ++k) { r[k] = zr[k]; r[NT + k] = zi[k]; }
        int mask = 16;
#pragma unroll
        for (int half = NT; half > 0; half >>= 1, mask >>= 1) {
            const bool up = (lane & mask) != 0;
#pragma unroll
            for (int i = 0; i < half; ++i) {
                const float away = up ? r[i] : r[i + half], own = up ? r[i + half] : r[i];
                r[i] = own + __shfl_xor_sync(0xffffffffu, away, mask);
            }
        }
#pragma unroll
        for (; mask > 0; mask >>= 1) r[0] += __shfl_xor_sync(0xffffffffu, r[0], mask);
        constexpr int kSpan = 32 / (2 * NT);
        const float mr = __shfl_sync(0xffffffffu, r[0], (lane % NT) * kSpan), mi = __shfl_sync(0xffffffffu, r[0], (NT + lane % NT) * kSpan);
        if (mine) {
            float a, in;
            lru_gate<T>(mr, mi, rb, ib, ns, us[lane * ld + o], a, in);
            const float st = fmaf(a, s_old, in);
            row[c] = st;
            out[static_cast<int64_t>(t) * sh.W + c] = from_float<T>(st * lru_gelu_of<T>(yv));
            if (sh.taps > 1) row[sh.W + static_cast<int64_t>(s_pos[lane] % sh.taps) * sh.W + c] = xv;
        }
    }
}

}  // namespace cvb

using namespace cvb;

static int lru_shape(LruShape& sh, int W, int parts, int taps, int stride, int y_off, int x_off, int64_t state_floats, int num_slots) {
    if (W <= 0 || parts <= 0 || taps <= 0 || num_slots <= 0) return CVB_E_SIZE;
    if (W % parts || y_off < 0 || x_off < 0 || stride < y_off + W || stride < x_off + W) return CVB_E_SHAPE;
    if (state_floats < static_cast<int64_t>(W) * (taps > 1 ? taps + 1 : 1)) return CVB_E_SHAPE;
    sh = LruShape{W, W / parts, taps, stride, y_off, x_off, state_floats, num_slots};
    return CVB_OK;
}

extern "C" int cvb_lru_conv(void* u, const void* packed, const float* bias_x, const float* conv_w, const float* conv_b, const float* state,
                            int64_t state_floats, int num_slots, const int* seq_of_token, const int* cu_seqlens, const int* state_slots,
                            const int* positions, int T, int W, int parts, int taps, int stride, int y_off, int x_off, int dtype, int* err_flag,
                            cudaStream_t stream) {
    if (T == 0) return CVB_OK;
    LruShape sh;
    const int rc = lru_shape(sh, W, parts, taps, stride, y_off, x_off, state_floats, num_slots);
    if (rc != CVB_OK || T < 0) return rc != CVB_OK ? rc : CVB_E_SIZE;
    const int n = dtype == CVB_DTYPE_BF16 ? 8 : 4;
    const bool vec = W % n == 0 && stride % n == 0 && x_off % n == 0 && ((reinterpret_cast<uintptr_t>(packed) | reinterpret_cast<uintptr_t>(u)) & 15) == 0;
    const int vcols = (W / n + kLruThreads - 1) / kLruThreads;
    int run = 8;                                        // shorter runs where long ones would leave SMs idle
    while (run > 2 && static_cast<int64_t>((T + run - 1) / run) * vcols < 592) run /= 2;
    const dim3 vgrid((T + run - 1) / run, vcols);
    if (vec && taps >= 2 && taps <= 4 && vgrid.y <= 65535) {
#define CALL_K(TY, K)                                                                                                         \
    launch_kernel(lru_conv_vec_kernel<TY, K>, vgrid, dim3(kLruThreads), 0, stream, (TY*)u, (const TY*)packed, bias_x, conv_w, conv_b, state, \
                  seq_of_token, cu_seqlens, state_slots, positions, T, run, sh, err_flag)
#define CALL(TY) if (taps == 4) { CALL_K(TY, 4); } else if (taps == 3) { CALL_K(TY, 3); } else { CALL_K(TY, 2); }
        CVB_DISPATCH_DTYPE(dtype, CALL);
#undef CALL
#undef CALL_K
        return launch_status();
    }
    const dim3 grid(T, min((W + kLruThreads - 1) / kLruThreads, 8));
#define CALL(TY)                                                                                                              \
    launch_kernel(lru_conv_kernel<TY>, grid, dim3(kLruThreads), 0, stream, (TY*)u, (const TY*)packed, bias_x, conv_w, conv_b, state, \
                  seq_of_token, cu_seqlens, state_slots, positions, sh, err_flag)
    CVB_DISPATCH_DTYPE(dtype, CALL);
#undef CALL
    return launch_status();
}

// `chunks`: how many chunks of `len` tokens the step's requests have together; `single`: no request has more than one (then
// `summary` is not used), otherwise `summary` holds 2 * W floats per chunk.
extern "C" int cvb_lru_scan(void* out, float* z, const void* u, const void* packed, const float* bias_y, const float* bias_x, const float* br,
                            const float* bi, const float* nsp, float* state, int64_t state_floats, int num_slots, float* summary,
                            int64_t summary_floats, const int* cu_seqlens, const int* state_slots, const int* positions, int S, int T,
                            int len, int chunks, int single, int W, int parts, int taps, int stride, int y_off, int x_off, int dtype,
                            int* err_flag, cudaStream_t stream) {
    if (T == 0 || S == 0) return CVB_OK;
    LruShape sh;
    const int rc = lru_shape(sh, W, parts, taps, stride, y_off, x_off, state_floats, num_slots);
    if (rc != CVB_OK) return rc;
    if (T < 0 || S < 0 || len <= 0 || chunks <= 0) return CVB_E_SIZE;
    if (!single && (summary == nullptr || summary_floats < static_cast<int64_t>(chunks) * 2 * W)) return CVB_E_SCRATCH;
    const dim3 grid(chunks, (W + kLruThreads - 1) / kLruThreads);
    if (grid.y > 65535) return CVB_E_SIZE;
#define CALL(TY)                                                                                                              \
    if (single) {                                                                                                             \
        launch_kernel(lru_finish_kernel<TY, true>, grid, dim3(kLruThreads), 0, stream, (TY*)out, z, (const TY*)u, (const TY*)packed, bias_y, \
                      bias_x, br, bi, nsp, state, summary, cu_seqlens, state_slots, positions, S, T, len, sh, err_flag);       \
    } else {                                                                                                                  \
        launch_kernel(lru_chunk_kernel<TY>, grid, dim3(kLruThreads), 0, stream, z, (const TY*)u, br, bi, nsp, state, summary,  \
                      cu_seqlens, state_slots, S, T, len, sh, err_flag);                                                      \
        launch_kernel(lru_finish_kernel<TY, false>, grid, dim3(kLruThreads), 0, stream, (TY*)out, z, (const TY*)u, (const TY*)packed, bias_y, \
                      bias_x, br, bi, nsp, state, summary, cu_seqlens, state_slots, positions, S, T, len, sh, err_flag);       \
    }
    CVB_DISPATCH_DTYPE(dtype, CALL);
#undef CALL
    return launch_status();
}

extern "C" int cvb_lru_step(void* out, const void* packed, const float* bias_y, const float* bias_x, const float* conv_w, const float* conv_b,
                            const void* gates, const float* br, const float* bi, const float* nsp, float* state, int64_t state_floats,
                            int num_slots, const int* cu_seqlens, const int* state_slots, const int* positions, int S, int W, int parts,
                            int taps, int stride, int y_off, int x_off, int dtype, int* err_flag, cudaStream_t stream) {
    if (S == 0) return CVB_OK;
    LruShape sh;
    const int rc = lru_shape(sh, W, parts, taps, stride, y_off, x_off, state_floats, num_slots);
    if (rc != CVB_OK) return rc;
    if (S < 0) return CVB_E_SIZE;
    // one channel a warp where that fills no more than two blocks per SM, else two or four
    int per_warp = 1;
    while (per_warp < 4 && static_cast<int64_t>(parts) * ((sh.part + kStepWarps * per_warp - 1) / (kStepWarps * per_warp)) > 296) per_warp *= 2;
    const int per_part = (sh.part + kStepWarps * per_warp - 1) / (kStepWarps * per_warp);
    const int nt = S <= 1 ? 1 : (S <= 2 ? 2 : (S <= 4 ? 4 : kStepTokens));
    const dim3 grid(parts * per_part, (S + nt - 1) / nt);
    const size_t smem = static_cast<size_t>(nt) * ((sh.part + 7) / 8 * 8) * sizeof(float);
    if (smem > 200 * 1024 || grid.y > 65535) return CVB_E_SIZE;
    const int vec = sh.part % 8 == 0 && (reinterpret_cast<uintptr_t>(gates) & 15) == 0;
#define CALL_NK(TY, NT, K)                                                                                                      \
    do {                                                                                                                      \
        if (smem > 48 * 1024) cudaFuncSetAttribute(lru_step_kernel<TY, NT, K>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);    \
        launch_kernel(lru_step_kernel<TY, NT, K>, grid, dim3(kStepThreads), smem, stream, (TY*)out, (const TY*)packed, bias_y, bias_x,     \
                      conv_w, conv_b, (const TY*)gates, br, bi, nsp, state, cu_seqlens, state_slots, positions, S, sh, vec, per_warp, err_flag);  \
    } while (0)
#define CALL_N(TY, NT) if (taps == 4) CALL_NK(TY, NT, 4); else CALL_NK(TY, NT, 0)
#define CALL(TY)                                                                                                              \
    if (nt == 1) { CALL_N(TY, 1); } else if (nt == 2) { CALL_N(TY, 2); } else if (nt == 4) { CALL_N(TY, 4); } else { CALL_N(TY, 8); }
    CVB_DISPATCH_DTYPE(dtype, CALL);
#undef CALL
#undef CALL_N
#undef CALL_NK
    return launch_status();
}
