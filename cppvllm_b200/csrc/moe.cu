// Routed feed-forward (mixture of experts): the router, the experts of a few tokens, and the experts of many.
//
//   route_topk     : z = x Wr^T + b in float (x may be bf16; Wr and b are float); top-k by z
//                    (of equal z the lower index first), weights exp(z_e) / sum over the k winners of exp(z_c):
//                    ids[t, k], weights[t, k], k in order of falling logit.
//                    `mode` 1: weights scale * exp(z_e) / sum over ALL experts of exp(z_c) instead (not renormalised over the
//                    winners).  Rows of Wr behind the E experts' (`extra` of them) are not experts: their raw products
//                    leave as extra_out[t, :] (a gate per token that shares the router's pass over x).
//                    `mode` 2: weights sigmoid(z_e) of the winners, each on its own (no sum over experts at all).
//                    `mode` 3: scores s = softmax(z) over all experts; the choice goes by s + bias (a correction that the weights
//                    do not see) among the experts of the `keep` groups (of `groups` equal groups of neighbours) whose largest
//                    choice score is largest; weights s_e / (sum over the winners of s_c + 1e-20).
//   Router outputs behind the E experts that have weights (`identity` of them) stand for the input itself: such a pair adds
//   weights[t, k] * x[t], touches no weights and gets no row in the sorted order.
//   With `on_input` = 1 a pair's weight multiplies the expert's INPUT instead of its output: y[t] = sum_k expert_e(T(w_k x[t])).
//   With `act` = 0 an expert is  Wd_e ( T(relu(T(Wu_e x))^2) )  and Wgu holds [E, ff, D];  with `act` = 2 it is
//   Wd_e ( T(g sigmoid(alpha g) (u + 1)) ),  g = min(Wg_e x, limit),  u = clamp(Wu_e x, -limit, limit).
//   An expert (`act` = 1) is  Wd_e ( T(silu(Wg_e x) * (Wu_e x)) ),  silu(z) = z * sigmoid(z);  the layer's output is
//   y[t] = T( sum_k weights[t, k] * expert_{ids[t, k]}(x[t]) ).  Wgu is [E, 2 ff, D] (gate rows over up rows), Wd is
//   [E, D, ff].  Products and the weighted sum are float; the gated activation is rounded to T once, as the input of a
//   product.
//   A few tokens (decode; also the float path): two kernels that read only the chosen experts' weights, which is what
//   bounds such a step, with the work of a (token, expert) pair spread over many blocks so that every SM streams:
//     expert_hidden : block (pair, slice of ff): a warp owns inner elements, its lanes a row of the gate and of the up weight
//     expert_down   : block (token, slice of D): walks the token's experts, a warp owns output elements
//   More tokens (bf16; from a handful of tokens that share experts up to prompt portions): the (token, expert) pairs are
//   sorted by expert on the device (sort_pairs_padded: counts, every expert's segment on a multiple of 128 rows, the
//   expert of every row tile; no trip to the host, so the step stays capturable), the tokens' rows are gathered into that
//   order, two grouped products run on the tcgen05 kernel (gemm_tcgen05.cu, grouped form: gate and up rows share a tile,
//   so the gated activation is the epilogue; every chosen expert's weights are read once, experts nobody chose cost
//   nothing), and combine_pairs adds a token's expert outputs up with its weights.
#include "common.cuh"

namespace cvb {

constexpr int kRouteWarps = 8;          // warps of a block, which share its tokens' rows out

// The choice from the logits z [E] (shared memory of the calling warp; in mode 3 with 2 E + groups floats): see the top of this file.
__device__ __forceinline__ void route_select(float* z, int* __restrict__ ids, float* __restrict__ weights, const float* __restrict__ bias,
                                             int64_t t, int E, int top, int mode, float scale, int groups, int keep, int lane) {
    float all = 0.f;                                    // modes 1 and 3: the sum over all experts, against the largest logit
    if (mode == 1 || mode == 3) {
        float big = -INFINITY;
        for (int e = lane; e < E; e += 32) big = fmaxf(big, z[e]);
        big = warp_max(big);
        for (int e = lane; e < E; e += 32) all += expf(z[e] - big);
        all = warp_sum(all);
        if (mode == 3) {
            float* s = z + E;                           // the scores; z becomes the choice scores
            float* best_of = s + E;                     // [groups] the largest choice score of each
            for (int e = lane; e < E; e += 32) {
                const float v = expf(z[e] - big) / all;
                s[e] = v;
                z[e] = v + (bias ? bias[e] : 0.f);
            }
            __syncwarp();
            const int per = E / groups;
            for (int g = lane; g < groups; g += 32) {
                float b = -INFINITY;
                for (int i = 0; i < per; ++i) b = fmaxf(b, z[g * per + i]);
                best_of[g] = b;
            }
            __syncwarp();
            // a group is left out if `keep` groups come before it (larger, or equal and in front)
            for (int e = lane; e < E; e += 32) {
                const int g = e / per;
                const float mine = best_of[g];
                int before = 0;
                for (int o = 0; o < groups; ++o) before += (best_of[o] > mine || (best_of[o] == mine && o < g)) ? 1 : 0;
                if (before >= keep) z[e] = -INFINITY;
            }
            __syncwarp();
        }
    }
    float z_first = 0.f, sum = 0.f;
    for (int k = 0; k < top; ++k) {
        float best = -INFINITY;
        int at = 0x7fffffff;
        for (int e = lane; e < E; e += 32) {
            const float v = z[e];
            if (v > best) { best = v; at = e; }          // the lower index wins among a lane's equals
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const int oa = __shfl_xor_sync(0xffffffffu, at, o);
            if (ob > best || (ob == best && oa < at)) { best = ob; at = oa; }
        }
        if (k == 0) z_first = best;
        if (mode == 3 && at >= E) at = 0;               // not reached: the kept groups hold `top` experts or more
        const float p = mode == 3 ? z[E + at] : (mode == 2 ? best : expf(best - z_first));      // mode 2 keeps the logit itself
        sum += p;
        if (lane == 0) {
            ids[t * top + k] = at;
            weights[t * top + k] = p;
            z[at] = -INFINITY;
        }
        __syncwarp();
    }
    if (mode == 2) {                                    // the winners' own logistic scores
        for (int k = lane; k < top; k += 32) weights[t * top + k] = scale / (1.f + expf(-weights[t * top + k]));
        return;
    }
    const float inv = mode == 1 ? scale / all : (mode == 3 ? scale / (sum + 1e-20f) : 1.f / sum);
    for (int k = lane; k < top; k += 32) weights[t * top + k] *= inv;     // lane 0's writes are visible after the syncwarp
}

// V elements of a row as floats: 16 bytes of weights, the matching activations
template <int V> __device__ __forceinline__ void route_load(const float* p, float (&f)[V]) {
    if constexpr (V == 4) { const float4 v = *reinterpret_cast<const float4*>(p); f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w; }
    else f[0] = p[0];
}
template <int V> __device__ __forceinline__ void route_load(const __nv_bfloat16* p, float (&f)[V]) {
    if constexpr (V == 4) {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
    } else f[0] = __bfloat162float(p[0]);
}

// A block takes NT tokens, its warps a slice of D each.  A warp holds the block's tokens by NE router outputs in registers, so a
// weight it loads serves NT tokens and an activation NE outputs; the warps' parts meet in shared memory in a fixed order.  NT = 8,
// NE = 4 for many tokens; NT = 1, NE = 16 for few (every row of the router in flight at once).
template <typename T, int V, int NT, int NE>
__global__ void __launch_bounds__(kRouteWarps * 32)
route_topk_kernel(int* __restrict__ ids, float* __restrict__ weights, const T* __restrict__ x, const float* __restrict__ wr,
                  const float* __restrict__ bias, int n_tokens, int D, int E, int top, int mode, float scale, int extra,
                  float* __restrict__ extra_out, int groups, int keep) {
    pdl_trigger();
    pdl_wait();
    constexpr int NV = NT * NE, kSpan = 32 / NV;        // sums per warp and round; lanes that end with the same one
    static_assert(NV == 16 || NV == 32, "a butterfly over the warp");
    extern __shared__ float smem[];                     // [NT][E] (mode 3: [..][2 E + groups]), then a round's parts
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int64_t t0 = static_cast<int64_t>(blockIdx.x) * NT;
    const int nt = static_cast<int>(n_tokens - t0 < NT ? n_tokens - t0 : NT), n_out = E + extra;
    const int per = mode == 3 ? 2 * E + groups : E;
    float* part = smem + NT * per;                      // [kRouteWarps][NV]
    const T* xr[NT];
#pragma unroll
    for (int k = 0; k < NT; ++k) xr[k] = x + (t0 + min(k, nt - 1)) * D;       // rows past the end repeat the last one
    for (int e0 = 0; e0 < n_out; e0 += NE) {
        const float* w = wr + static_cast<int64_t>(e0) * D;
        float r[NV];                                    // [token][output]
#pragma unroll
        for (int i = 0; i < NV; ++i) r[i] = 0.f;
#pragma unroll 2
        for (int i = (warp * 32 + lane) * V; i < D; i += kRouteWarps * 32 * V) {
            float wv[NE][V];
#pragma unroll
            for (int q = 0; q < NE; ++q) {
                if (e0 + q < n_out) route_load<V>(w + static_cast<int64_t>(q) * D + i, wv[q]);
                else {
#pragma unroll
                    for (int v = 0; v < V; ++v) wv[q][v] = 0.f;
                }
            }
#pragma unroll
            for (int k = 0; k < NT; ++k) {
                float xv[V];
                route_load<V>(xr[k] + i, xv);
#pragma unroll
                for (int q = 0; q < NE; ++q)
#pragma unroll
                    for (int v = 0; v < V; ++v) r[k * NE + q] = fmaf(xv[v], wv[q][v], r[k * NE + q]);
            }
        }
        // NV sums over 32 lanes by a transposing butterfly: lane l ends with sum l / kSpan
        int mask = 16;
#pragma unroll
        for (int half = NV / 2; half > 0; half >>= 1, mask >>= 1) {
            const bool up = (lane & mask) != 0;
#pragma unroll
            for (int i = 0; i < half; ++i) {
                const float away = up ? r[i] : r[i + half], own = up ? r[i + half] : r[i];
                r[i] = own + __shfl_xor_sync(0xffffffffu, away, mask);
            }
        }
#pragma unroll
        for (; mask > 0; mask >>= 1) r[0] += __shfl_xor_sync(0xffffffffu, r[0], mask);
        __syncthreads();                                // the round before has been read
        if (lane % kSpan == 0) part[warp * NV + lane / kSpan] = r[0];
        __syncthreads();
        if (warp == 0 && lane < NV) {
            float v = 0.f;
#pragma unroll
            for (int g = 0; g < kRouteWarps; ++g) v += part[g * NV + lane];
            const int k = lane / NE, e = e0 + lane % NE;
            if (k < nt && e < n_out) {
                if (e < E) smem[k * per + e] = v + (bias && mode != 3 ? bias[e] : 0.f);
                else extra_out[(t0 + k) * extra + (e - E)] = v;
            }
        }
    }
    __syncthreads();
    for (int k = warp; k < nt; k += kRouteWarps) route_select(smem + k * per, ids, weights, bias, t0 + k, E, top, mode, scale, groups, keep, lane);
}

constexpr int kExpertThreads = 256;
constexpr int kExpertWarps = kExpertThreads / 32;

template <typename T> __device__ __forceinline__ float silu_exact(float g) { return g / (1.f + expf(-g)); }

// Eight weights of a bf16 row against eight floats in shared memory: one 16-byte load per lane and row.
__device__ __forceinline__ float dot8(const __nv_bfloat16* __restrict__ w, const float* __restrict__ xs, float acc) {
    const uint4 raw = *reinterpret_cast<const uint4*>(w);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
    const float4 x0 = *reinterpret_cast<const float4*>(xs), x1 = *reinterpret_cast<const float4*>(xs + 4);
    float2 f = __bfloat1622float2(h[0]);
    acc = fmaf(x0.x, f.x, acc); acc = fmaf(x0.y, f.y, acc);
    f = __bfloat1622float2(h[1]);
    acc = fmaf(x0.z, f.x, acc); acc = fmaf(x0.w, f.y, acc);
    f = __bfloat1622float2(h[2]);
    acc = fmaf(x1.x, f.x, acc); acc = fmaf(x1.y, f.y, acc);
    f = __bfloat1622float2(h[3]);
    acc = fmaf(x1.z, f.x, acc); acc = fmaf(x1.w, f.y, acc);
    return acc;
}
template <typename T> __device__ __forceinline__ bool rows_by_16_bytes(const T*, int) { return false; }
template <> __device__ __forceinline__ bool rows_by_16_bytes<__nv_bfloat16>(const __nv_bfloat16* base, int row_len) {
    return row_len % 8 == 0 && (reinterpret_cast<uintptr_t>(base) & 15) == 0;
}
template <typename T> __device__ __forceinline__ float dot8_of(const T*, const float*, float acc) { return acc; }
template <> __device__ __forceinline__ float dot8_of<__nv_bfloat16>(const __nv_bfloat16* w, const float* xs, float acc) { return dot8(w, xs, acc); }

constexpr int kActRelu2 = 0, kActClamped = 2;            // 1: silu

__device__ __forceinline__ float gated_of(float g, float u, int act, float limit, float alpha) {
    if (act == kActClamped) {
        g = fminf(g, limit);
        u = fminf(fmaxf(u, -limit), limit);
        return g * (1.f / (1.f + expf(-alpha * g))) * (u + 1.f);
    }
    return silu_exact<float>(g) * u;
}

// hid[pair, f] = T(silu(Wg_e[f] . x) * (Wu_e[f] . x)) for the block's slice of f; pair = t * top + k, e = ids[pair]
template <typename T>
__global__ void __launch_bounds__(kExpertThreads)
expert_hidden_kernel(T* __restrict__ hid, const T* __restrict__ x, const int* __restrict__ ids, const T* __restrict__ wgu,
                     int D, int F, int E, int top, int per_block, int act, const float* __restrict__ in_weights,
                     int identity, float limit, float alpha, int* __restrict__ err) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) float smem[];
    float* xs = smem;                                   // [D]
    const int64_t pair = blockIdx.x;
    const int64_t t = pair / top;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    int e = ids[pair];
    if (e >= E && e < E + identity) return;             // the input itself: nothing to compute here
    if (e < 0 || e >= E) {
        if (threadIdx.x == 0) atomicExch(err, 7);
        e = 0;
    }
    const bool gated = act != kActRelu2;
    const float wi = in_weights != nullptr ? in_weights[pair] : 1.f;
    if (in_weights != nullptr) {
        for (int i = threadIdx.x; i < D; i += kExpertThreads) xs[i] = rnd<T>(wi * to_float(x[t * D + i]));
    } else {
        for (int i = threadIdx.x; i < D; i += kExpertThreads) xs[i] = to_float(x[t * D + i]);
    }
    __syncthreads();
    const T* g_rows = wgu + static_cast<int64_t>(e) * (gated ? 2 : 1) * F * D;
    const T* u_rows = g_rows + static_cast<int64_t>(F) * D;
    const int f0 = blockIdx.y * per_block, f1 = min(F, f0 + per_block);
    const bool wide = rows_by_16_bytes<T>(wgu, D);
    for (int f = f0 + warp; f < f1; f += kExpertWarps) {
        const T* gr = g_rows + static_cast<int64_t>(f) * D;
        const T* ur = u_rows + static_cast<int64_t>(f) * D;
        float g = 0.f, u = 0.f;
        if (gated) {
            if (wide) {
                for (int i = lane * 8; i < D; i += 256) { g = dot8_of<T>(gr + i, xs + i, g); u = dot8_of<T>(ur + i, xs + i, u); }
            } else {
                for (int i = lane; i < D; i += 32) {
                    const float xv = xs[i];
                    g = fmaf(xv, to_float(gr[i]), g);
                    u = fmaf(xv, to_float(ur[i]), u);
                }
            }
            g = warp_sum(g);
            u = warp_sum(u);
            if (lane == 0) hid[pair * F + f] = from_float<T>(gated_of(g, u, act, limit, alpha));
        } else {
            if (wide) {
                for (int i = lane * 8; i < D; i += 256) g = dot8_of<T>(gr + i, xs + i, g);
            } else {
                for (int i = lane; i < D; i += 32) g = fmaf(xs[i], to_float(gr[i]), g);
            }
            g = fmaxf(rnd<T>(warp_sum(g)), 0.f);
            if (lane == 0) hid[pair * F + f] = from_float<T>(g * g);
        }
    }
}

// y[t, d] = T(sum_k weights[t, k] * (Wd_e[d] . hid[t * top + k])) for the block's slice of d
template <typename T>
__global__ void __launch_bounds__(kExpertThreads)
expert_down_kernel(T* __restrict__ y, const T* __restrict__ hid, const T* __restrict__ x, const int* __restrict__ ids,
                   const float* __restrict__ weights, const T* __restrict__ wd, int D, int F, int E, int top, int per_block, int on_input,
                   int identity) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) float smem[];
    float* hs = smem;                                   // [F]
    float* acc = hs + F;                                // [per_block]
    const int64_t t = blockIdx.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int d0 = blockIdx.y * per_block, d1 = min(D, d0 + per_block);
    for (int i = threadIdx.x; i < per_block; i += kExpertThreads) acc[i] = 0.f;
    __syncthreads();                                    // an identity expert adds before any other barrier
    const bool wide = rows_by_16_bytes<T>(wd, F);
    for (int k = 0; k < top; ++k) {
        int e = ids[t * top + k];
        const float wk = on_input ? 1.f : weights[t * top + k];
        if (e >= E && e < E + identity) {                // the input itself, times the weight
            for (int d = d0 + warp; d < d1; d += kExpertWarps)
                if (lane == 0) acc[d - d0] = fmaf(weights[t * top + k], to_float(x[t * D + d]), acc[d - d0]);
            continue;
        }
        if (e < 0 || e >= E) e = 0;                      // reported by the kernel in front
        __syncthreads();
        for (int i = threadIdx.x; i < F; i += kExpertThreads) hs[i] = to_float(hid[(t * top + k) * F + i]);
        __syncthreads();
        const T* d_rows = wd + static_cast<int64_t>(e) * D * F;
        for (int d = d0 + warp; d < d1; d += kExpertWarps) {
            const T* dr = d_rows + static_cast<int64_t>(d) * F;
            float o = 0.f;
            if (wide) {
                for (int i = lane * 8; i < F; i += 256) o = dot8_of<T>(dr + i, hs + i, o);
            } else {
                for (int i = lane; i < F; i += 32) o = fmaf(hs[i], to_float(dr[i]), o);
            }
            o = warp_sum(o);
            if (lane == 0) acc[d - d0] = fmaf(wk, o, acc[d - d0]);     // a warp owns its d: no other warp touches acc[d - d0]
        }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < d1 - d0; i += kExpertThreads) y[t * D + d0 + i] = from_float<T>(acc[i]);
}

// ---- many tokens: pairs sorted by expert, grouped products on the tensor cores ------------------------------------------

constexpr int kSortThreads = 1024;

// Counts per expert, then every expert's segment of sorted rows, which starts on a multiple of `pad` rows (the tcgen05
// grouped product's row tiles are 128 rows of ONE expert).  One block.  The order of an expert's rows among themselves
// is not fixed; no result depends on it.  tile_expert[i]: the expert of row tile i, -1 for tiles behind the last segment (max_tiles
// entries).  row_token[slot]: the token whose row goes to sorted row `slot` (0 for the padding rows: they are computed
// and never read).  slot_of[pair]: where the pair's row lies; -1 for a pair whose expert is the input itself.
__global__ void __launch_bounds__(kSortThreads)
sort_pairs_padded_kernel(int* __restrict__ tile_expert, int* __restrict__ row_token, int* __restrict__ slot_of,
                         const int* __restrict__ ids, int n_pairs, int E, int top, int pad, int max_tiles, int identity,
                         int* __restrict__ err) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ int ismem[];
    int* count = ismem;                                 // [E]
    int* start = count + E;                             // [E + 1]
    for (int e = threadIdx.x; e < E; e += kSortThreads) count[e] = 0;
    for (int i = threadIdx.x; i < max_tiles * pad; i += kSortThreads) row_token[i] = 0;
    __syncthreads();
    for (int i = threadIdx.x; i < n_pairs; i += kSortThreads) {
        int e = ids[i];
        if (e >= E && e < E + identity) continue;
        if (e < 0 || e >= E) { atomicExch(err, 7); e = 0; }
        atomicAdd(&count[e], 1);
    }
    __syncthreads();
    if (threadIdx.x == 0) {
        int run = 0;
        for (int e = 0; e < E; ++e) { start[e] = run; run += (count[e] + pad - 1) / pad * pad; }
        start[E] = run;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < max_tiles; i += kSortThreads) {
        int e = -1;
        if (i * pad < start[E]) {
            int lo = 0, hi = E - 1;                      // the last expert whose segment starts at or before the tile
            while (lo < hi) {
                const int mid = (lo + hi + 1) >> 1;
                if (start[mid] <= i * pad) lo = mid; else hi = mid - 1;
            }
            e = lo;
            while (e < E - 1 && start[e + 1] <= i * pad) ++e;      // empty experts share a start: take the one that has rows
        }
        tile_expert[i] = e;
    }
    for (int e = threadIdx.x; e < E; e += kSortThreads) count[e] = 0;
    __syncthreads();
    for (int i = threadIdx.x; i < n_pairs; i += kSortThreads) {
        int e = ids[i];
        if (e >= E && e < E + identity) { slot_of[i] = -1; continue; }
        if (e < 0 || e >= E) e = 0;
        const int slot = start[e] + atomicAdd(&count[e], 1);
        row_token[slot] = i / top;
        slot_of[i] = slot;
    }
}

// xs[slot_of[pair], :] = T(weights[pair] * x[pair / top, :]): the rows of the grouped product when a pair's weight multiplies
// the expert's input.  Padding rows keep what they held; they are computed and never read.
__global__ void scatter_pairs_scaled_kernel(__nv_bfloat16* __restrict__ xs, const __nv_bfloat16* __restrict__ x,
                                            const int* __restrict__ slot_of, const float* __restrict__ weights, int D, int top) {
    pdl_trigger();
    pdl_wait();
    const int64_t pair = blockIdx.x;
    const float w = weights[pair];
    if (slot_of[pair] < 0) return;
    const __nv_bfloat16* src = x + pair / top * D;
    __nv_bfloat16* dst = xs + static_cast<int64_t>(slot_of[pair]) * D;
    for (int d = threadIdx.x; d < D; d += blockDim.x) dst[d] = __float2bfloat16_rn(w * __bfloat162float(src[d]));
}

// y[t, :] = sum_k weights[t, k] * rows[slot_of[t * top + k], :]   (weights = nullptr: all 1; a negative slot: x[t, :] instead)
__global__ void combine_pairs_kernel(__nv_bfloat16* __restrict__ y, const __nv_bfloat16* __restrict__ rows, const __nv_bfloat16* __restrict__ x,
                                     const int* __restrict__ slot_of, const float* __restrict__ weights, int D, int top) {
    pdl_trigger();
    pdl_wait();
    const int64_t t = blockIdx.x;
    for (int d = threadIdx.x; d < D; d += blockDim.x) {
        float s = 0.f;
        for (int k = 0; k < top; ++k) {
            const int64_t slot = slot_of[t * top + k];
            s = fmaf(weights != nullptr ? weights[t * top + k] : 1.f, __bfloat162float(slot >= 0 ? rows[slot * D + d] : x[t * D + d]), s);
        }
        y[t * D + d] = __float2bfloat16_rn(s);
    }
}

}  // namespace cvb

using namespace cvb;

extern "C" int cvb_route_topk(int* ids, float* weights, const void* x, const float* wr, const float* bias, int T, int D, int E,
                              int top, int mode, float scale, int extra, float* extra_out, int groups, int keep, int dtype,
                              cudaStream_t stream) {
    if (T == 0) return CVB_OK;
    if (T < 0 || D <= 0 || E <= 0 || top <= 0 || extra < 0 || (extra > 0 && extra_out == nullptr)) return CVB_E_SIZE;
    if (mode < 0 || mode > 3) return CVB_E_SHAPE;
    if (top > E || E > 2048) return CVB_E_SHAPE;
    if (mode == 3 && (groups <= 0 || E % groups || keep <= 0 || keep > groups || top > keep * (E / groups))) return CVB_E_SHAPE;
    const bool few = T <= 512;
    const int nt = few ? 1 : 8;
    const size_t smem = (static_cast<size_t>(nt) * (mode == 3 ? 2 * E + groups : E) + kRouteWarps * 32) * sizeof(float);
    if (smem > 200 * 1024) return CVB_E_SIZE;
    const bool four = D % 4 == 0 && ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(wr)) & 15) == 0;
#define CALL_N(TY, V, NT, NE)                                                                                                 \
    do {                                                                                                                      \
        if (smem > 48 * 1024) cudaFuncSetAttribute(route_topk_kernel<TY, V, NT, NE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        launch_kernel(route_topk_kernel<TY, V, NT, NE>, dim3((T + NT - 1) / NT), dim3(kRouteWarps * 32), smem, stream, ids, weights,  \
                      (const TY*)x, wr, bias, T, D, E, top, mode, scale, extra, extra_out, groups, keep);                       \
    } while (0)
#define CALL_V(TY, V) if (few) CALL_N(TY, V, 1, 16); else CALL_N(TY, V, 8, 4)
#define CALL(TY) if (four) { CALL_V(TY, 4); } else { CALL_V(TY, 1); }
    CVB_DISPATCH_DTYPE(dtype, CALL);
#undef CALL
#undef CALL_V
#undef CALL_N
    return launch_status();
}

extern "C" int cvb_expert_rows(void* y, void* hid, const void* x, const int* ids, const float* weights, const void* wgu,
                               const void* wd, int T, int D, int F, int E, int top, int act, int on_input, int identity, float limit,
                               float alpha, int dtype, int* err_flag, cudaStream_t stream) {
    if (T == 0) return CVB_OK;
    if (T < 0 || D <= 0 || F <= 0 || E <= 0 || top <= 0 || identity < 0) return CVB_E_SIZE;
    if (act < kActRelu2 || act > kActClamped) return CVB_E_SHAPE;
    if (static_cast<size_t>(D) * sizeof(float) > 160 * 1024 || static_cast<size_t>(F) * sizeof(float) > 160 * 1024) return CVB_E_SIZE;
    // slices sized so that a step of one token still gives every SM a block or two
    const int64_t pairs = static_cast<int64_t>(T) * top;
    int f_per = kExpertWarps;
    while (pairs * ((F + f_per - 1) / f_per) > 1184 && f_per < F) f_per *= 2;
    int d_per = kExpertWarps;
    while (static_cast<int64_t>(T) * ((D + d_per - 1) / d_per) > 1184 && d_per < D) d_per *= 2;
    const size_t smem1 = static_cast<size_t>(D) * sizeof(float);
    const size_t smem2 = (static_cast<size_t>(F) + d_per) * sizeof(float);
    if (pairs > 2147483647LL / 2 || smem2 > 200 * 1024) return CVB_E_SIZE;
#define CALL(TY)                                                                                                         \
    do {                                                                                                                 \
        if (smem1 > 48 * 1024)                                                                                           \
            cudaFuncSetAttribute(expert_hidden_kernel<TY>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem1);     \
        if (smem2 > 48 * 1024)                                                                                           \
            cudaFuncSetAttribute(expert_down_kernel<TY>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem2);       \
        launch_kernel(expert_hidden_kernel<TY>, dim3((unsigned)pairs, (F + f_per - 1) / f_per), dim3(kExpertThreads), smem1,  \
                      stream, (TY*)hid, (const TY*)x, ids, (const TY*)wgu, D, F, E, top, f_per, act, on_input ? weights : nullptr, identity, limit, alpha, err_flag); \
        launch_kernel(expert_down_kernel<TY>, dim3(T, (D + d_per - 1) / d_per), dim3(kExpertThreads), smem2, stream,      \
                      (TY*)y, (const TY*)hid, (const TY*)x, ids, weights, (const TY*)wd, D, F, E, top, d_per, on_input, identity);    \
    } while (0)
    CVB_DISPATCH_DTYPE(dtype, CALL);
#undef CALL
    return launch_status();
}

// Sorts the pairs for the tcgen05 grouped product (see sort_pairs_padded_kernel); max_tiles * 128 rows of scratch.
extern "C" int cvb_sort_pairs_padded(int* tile_expert, int* row_token, int* slot_of, const int* ids, int T, int E, int top,
                                     int max_tiles, int identity, int* err_flag, cudaStream_t stream) {
    if (T <= 0 || E <= 0 || top <= 0 || max_tiles <= 0 || E > 4096) return CVB_E_SIZE;
    const int64_t pairs = static_cast<int64_t>(T) * top;
    if (pairs > (1 << 30) || (pairs + 127) / 128 + E > max_tiles) return CVB_E_SCRATCH;
    launch_kernel(sort_pairs_padded_kernel, dim3(1), dim3(kSortThreads), (2 * static_cast<size_t>(E) + 1) * sizeof(int), stream,
                  tile_expert, row_token, slot_of, ids, static_cast<int>(pairs), E, top, 128, max_tiles, identity, err_flag);
    return launch_status();
}

extern "C" int cvb_scatter_pairs_scaled_bf16(void* xs, const void* x, const int* slot_of, const float* weights, int T, int D, int top,
                                             cudaStream_t stream) {
    if (T <= 0 || D <= 0 || top <= 0) return CVB_E_SIZE;
    launch_kernel(scatter_pairs_scaled_kernel, dim3(static_cast<unsigned>(T) * top), dim3(D >= 1024 ? 256 : 128), 0, stream,
                  (__nv_bfloat16*)xs, (const __nv_bfloat16*)x, slot_of, weights, D, top);
    return launch_status();
}

extern "C" int cvb_combine_pairs_bf16(void* y, const void* rows, const void* x, const int* slot_of, const float* weights, int T, int D, int top,
                                      cudaStream_t stream) {
    if (T <= 0 || D <= 0 || top <= 0) return CVB_E_SIZE;
    launch_kernel(combine_pairs_kernel, dim3(T), dim3(D >= 1024 ? 256 : 128), 0, stream, (__nv_bfloat16*)y,
                  (const __nv_bfloat16*)rows, (const __nv_bfloat16*)x, slot_of, weights, D, top);
    return launch_status();
}
