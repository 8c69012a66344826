// Mixture-of-experts feed-forward of layered decoders.
//
//   moe_route         fp32 router: z = W_r h, s = softmax(z) over all n routed outputs (the last n_identity of them are identity
//                     experts: output = input); choice = s + correction; the n outputs form `groups` equal groups of
//                     neighbours, a group scores its largest choice (or the sum of its two largest), only the best `keep` groups stay eligible; the `top`
//                     largest eligible choices are taken, each weighted by its s, optionally divided by the sum of the chosen ones' s.  Ties go to the lower index.
//                     Another form chooses by z (+ a bias) itself and weights by the softmax over the chosen z alone.
//                     One more output may gate a shared expert (its sigmoid, not routed).  Writes the dense weights [T, n] (0 where not chosen) and the chosen (index, weight) pairs [T, top].
//   moe_gateup_sparse / moe_down_sparse   few tokens (decode): one CTA column per (token, chosen expert) streams only that
//                     expert's rows: act = silu(W_gate h) * (W_up h), then y = sum_k w_k W_down[e_k] act_k + (identity weights) h
//   moe_gateup_mma / moe_down_mma   the same for 2 to 16 tokens in bf16 on tensor cores, expert by expert: a weight that several tokens chose is read once
//   rows_axpy         y[t] += (sum of the identity weights of t) * h[t]       (after the dense, masked form for prompts)
//
// Weights are packed: w13 [E * 2 * ff, width] with rows (2c, 2c + 1) = (gate_c, up_c) of each expert in turn; w2 [width, E * ff]
// with expert e's down projection in columns e*ff .. (e+1)*ff - 1.  Prompts run the dense form through the Linear kernels:
// every expert on every token, the SwiGLU epilogue multiplying by the token's routing weight of the column's expert.
#pragma once
#include "hybrid_common.cuh"

namespace mbh {

struct MoeRouteArgs {
    const void* h;            // [T, width]
    const void* w_router;     // [n, width]
    const void* correction;   // [n] or null
    float* dense;             // [T, n + always]
    int* idx;                 // [T, top + always]
    float* wsel;              // [T, top + always]
    int width, n, groups, keep, top;
    int score;                // 0: softmax over the outputs; 1: sigmoid of each output; 2: the outputs themselves decide (one group), the
                              // weights are the softmax over the chosen ones alone
    const void* w_bias;       // [n] or null: added to the outputs before anything else
    float scale;              // the weights (dense and wsel) are the chosen scores times this
    int group_two;            // a group scores the sum of its two largest choices instead of its largest
    int renorm;               // the weights are divided by (the sum of the chosen scores + 1e-20)
    const void* w_gate;       // [width] or null: one more output whose sigmoid gates a shared expert ...
    float* gate;              // [T] ... goes here; it takes no part in the routing
    int always;               // experts n .. n + always - 1 take no part in the routing either: every token has them, with weight 1
};

// (value, index) argmax over a warp; the lower index wins a tie
__device__ __forceinline__ void warp_argmax(float& v, int& i) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, v, o);
        const int oi = __shfl_xor_sync(0xffffffffu, i, o);
        if (ov > v || (ov == v && oi < i)) { v = ov; i = oi; }
    }
}

// dot product of two rows of K elements over a warp (16-byte loads when both rows allow it); every lane gets the sum
template <typename T>
__device__ __forceinline__ float warp_dot(const T* __restrict__ w, const T* __restrict__ x, int K, int lane) {
    constexpr int V = Vec<T>::N;
    float acc = 0.f;
    if (K % V == 0 && ((reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(x)) % 16 == 0)) {
        for (int k = lane * V; k < K; k += 32 * V) {
            float wv[V], xv[V];
            Vec<T>::load(w + k, wv);
            Vec<T>::load(x + k, xv);
#pragma unroll
            for (int i = 0; i < V; ++i) acc = fmaf(wv[i], xv[i], acc);
        }
    } else {
        for (int k = lane; k < K; k += 32) acc = fmaf(to_f(w[k]), to_f(x[k]), acc);
    }
    return warp_sum(acc);
}

constexpr int MOE_ROUTE_THREADS = 256;

// one CTA per token; shared memory: z[n] | choice[n] | gbest[groups] | kept[groups]
template <typename T>
__global__ void __launch_bounds__(MOE_ROUTE_THREADS) moe_route_kernel(MoeRouteArgs a) {
    extern __shared__ float sm[];
    float* z = sm;
    float* ch = sm + a.n;
    float* gb = sm + 2 * a.n;
    float* kept = gb + a.groups;
    const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
    const T* h = static_cast<const T*>(a.h) + (size_t)t * a.width;
    const T* W = static_cast<const T*>(a.w_router);
    for (int e = warp; e < a.n + (a.w_gate ? 1 : 0); e += nw) {
        const float acc = warp_dot<T>(e < a.n ? W + (size_t)e * a.width : static_cast<const T*>(a.w_gate), h, a.width, lane);
        if (lane == 0) {
            if (e < a.n) z[e] = acc + (a.w_bias ? to_f(static_cast<const T*>(a.w_bias)[e]) : 0.f);
            else a.gate[t] = sigmoid_exact(acc);
        }
    }
    __syncthreads();
    if (warp != 0) return;
    const int dn = a.n + a.always, tk = a.top + a.always;
    for (int s = lane; s < a.always; s += 32) {
        a.dense[(size_t)t * dn + a.n + s] = 1.f;
        a.idx[(size_t)t * tk + a.top + s] = a.n + s;
        a.wsel[(size_t)t * tk + a.top + s] = 1.f;
    }
    float sum = 1.f;
    if (a.score == 2) {
        float mx = -INFINITY;  // the largest output is always chosen: it keeps the exponentials of the chosen ones in range
        for (int e = lane; e < a.n; e += 32) { mx = fmaxf(mx, z[e]); ch[e] = z[e]; a.dense[(size_t)t * dn + e] = 0.f; }
        mx = warp_max(mx);
        __syncwarp();
        float den = 0.f;
        for (int k = 0; k < a.top; ++k) {
            float v = -INFINITY; int ei = 0x7fffffff;
            for (int e = lane; e < a.n; e += 32)
                if (ch[e] > v) { v = ch[e]; ei = e; }
            warp_argmax(v, ei);
            if (ei == 0x7fffffff) ei = 0;
            den += expf(v - mx);
            if (lane == 0) { a.idx[(size_t)t * tk + k] = ei; ch[ei] = -INFINITY; }
            __syncwarp();
        }
        for (int k = lane; k < a.top; k += 32) {
            const int ei = a.idx[(size_t)t * tk + k];
            const float w = expf(z[ei] - mx) / den * a.scale;
            a.wsel[(size_t)t * tk + k] = w;
            a.dense[(size_t)t * dn + ei] = w;
        }
        return;
    }
    if (a.score == 1) {
        for (int e = lane; e < a.n; e += 32) z[e] = sigmoid_exact(z[e]);
    } else {
        float mx = -INFINITY;
        for (int e = lane; e < a.n; e += 32) mx = fmaxf(mx, z[e]);
        mx = warp_max(mx);
        sum = 0.f;
        for (int e = lane; e < a.n; e += 32) { const float p = expf(z[e] - mx); z[e] = p; sum += p; }
        sum = warp_sum(sum);
    }
    const T* corr = static_cast<const T*>(a.correction);
    for (int e = lane; e < a.n; e += 32) {
        const float s = z[e] / sum;
        z[e] = s;
        ch[e] = s + (corr ? to_f(corr[e]) : 0.f);
        a.dense[(size_t)t * dn + e] = 0.f;
    }
    __syncwarp();
    if (a.groups > 1 && a.keep < a.groups) {
        const int gs = a.n / a.groups;
        for (int g = lane; g < a.groups; g += 32) {
            float b = -INFINITY, b2 = -INFINITY;
            for (int e = g * gs; e < (g + 1) * gs; ++e) {
                b2 = fmaxf(b2, fminf(b, ch[e]));
                b = fmaxf(b, ch[e]);
            }
            gb[g] = (a.group_two && gs > 1) ? b + b2 : b;
            kept[g] = 0.f;
        }
        __syncwarp();
        // take the best `keep` groups one at a time; then drop the experts of the others
        for (int k = 0; k < a.keep; ++k) {
            float v = -INFINITY; int gi = 0x7fffffff;
            for (int g = lane; g < a.groups; g += 32)
                if (kept[g] == 0.f && (gi == 0x7fffffff || gb[g] > v)) { v = gb[g]; gi = g; }
            warp_argmax(v, gi);
            if (lane == 0 && gi != 0x7fffffff) kept[gi] = 1.f;
            __syncwarp();
        }
        for (int e = lane; e < a.n; e += 32)
            if (kept[e / gs] == 0.f) ch[e] = -INFINITY;
        __syncwarp();
    }
    float total = 0.f;  // of the chosen scores, the same in every lane
    for (int k = 0; k < a.top; ++k) {
        float v = -INFINITY; int ei = 0x7fffffff;
        for (int e = lane; e < a.n; e += 32)
            if (ch[e] > v) { v = ch[e]; ei = e; }
        warp_argmax(v, ei);
        if (ei == 0x7fffffff) ei = 0;  // fewer eligible outputs than `top` (a configuration error): weight 0 below
        const float w = (v == -INFINITY) ? 0.f : z[ei];
        total += w;
        if (lane == 0) {
            a.idx[(size_t)t * tk + k] = ei;
            a.wsel[(size_t)t * tk + k] = w * a.scale;
            if (v != -INFINITY) { a.dense[(size_t)t * dn + ei] = w * a.scale; ch[ei] = -INFINITY; }
        }
        __syncwarp();
    }
    if (a.renorm) {  // every value was written by this warp; the barrier above ordered the writes
        const float den = total + 1e-20f;
        for (int k = lane; k < a.top; k += 32) {
            const int ei = a.idx[(size_t)t * tk + k];
            const float w = z[ei] / den * a.scale;
            a.wsel[(size_t)t * tk + k] = w;
            a.dense[(size_t)t * dn + ei] = w;
        }
    }
}

struct MoeSparseArgs {
    const void* h;            // [T, width]
    const void* w13;          // [E * 2 * ff, width]
    const void* w2;           // [width, E * ff]
    const int* idx;           // [T, top]
    const float* wsel;        // [T, top]
    void* act;                // [T * top, ff]
    float* y32;               // [T, width]
    int width, ff, E, top;
    int glu;                  // 0: silu(gate) * up, the routing weight multiplies the expert's OUTPUT; 1: the weight multiplies the
    float limit, alpha;       //    expert's INPUT: g = min(w gate, limit), u = clamp(w up, +-limit), act = g sigmoid(alpha g) (u + 1);
                              // 2: experts without a gate, act = max(W_up h, 0)^2, w13 = [E * ff, width] plain rows, weight on the OUTPUT
    int accumulate;           // y32 += the experts' sum (y32 is the residual stream) instead of y32 = it
};

constexpr int MOE_WARPS = 8;

// grid (ceil(ff / MOE_WARPS), T * top): a warp per hidden unit of the chosen expert
template <typename T>
__global__ void __launch_bounds__(MOE_WARPS * 32) moe_gateup_sparse_kernel(MoeSparseArgs a) {
    const int slot = blockIdx.y, t = slot / a.top, e = a.idx[slot];
    if (e >= a.E) return;  // identity expert: no weights
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, c = blockIdx.x * MOE_WARPS + warp;
    if (c >= a.ff) return;
    const T* h = static_cast<const T*>(a.h) + (size_t)t * a.width;
    if (a.glu == 2) {
        const float u = rnd<T>(warp_dot<T>(static_cast<const T*>(a.w13) + ((size_t)e * a.ff + c) * a.width, h, a.width, lane));
        if (lane == 0) { const float r = fmaxf(u, 0.f); static_cast<T*>(a.act)[(size_t)slot * a.ff + c] = from_f<T>(r * r); }
        return;
    }
    const T* wg = static_cast<const T*>(a.w13) + ((size_t)e * a.ff + c) * 2 * a.width;
    float g = rnd<T>(warp_dot<T>(wg, h, a.width, lane)), u = rnd<T>(warp_dot<T>(wg + a.width, h, a.width, lane));
    if (lane != 0) return;
    float act;
    if (a.glu == 1) {
        const float w = a.wsel[slot];
        g = fminf(g * w, a.limit);
        u = fminf(fmaxf(u * w, -a.limit), a.limit);
        act = g * sigmoid_exact(a.alpha * g) * (u + 1.f);
    } else {
        act = g * sigmoid_exact(g) * u;
    }
    static_cast<T*>(a.act)[(size_t)slot * a.ff + c] = from_f<T>(act);
}

// grid (ceil(width / MOE_WARPS), T): a warp per output column, summing the token's chosen experts in slot order
template <typename T>
__global__ void __launch_bounds__(MOE_WARPS * 32) moe_down_sparse_kernel(MoeSparseArgs a) {
    const int t = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n = blockIdx.x * MOE_WARPS + warp;
    if (n >= a.width) return;
    const T* wrow = static_cast<const T*>(a.w2) + (size_t)n * a.E * a.ff;
    float acc = 0.f;
    for (int k = 0; k < a.top; ++k) {
        const int slot = t * a.top + k, e = a.idx[slot];
        const float w = a.glu == 1 ? 1.f : a.wsel[slot];
        if (e >= a.E) acc += a.wsel[slot] * to_f(static_cast<const T*>(a.h)[(size_t)t * a.width + n]);
        else acc += w * rnd<T>(warp_dot<T>(wrow + (size_t)e * a.ff, static_cast<const T*>(a.act) + (size_t)slot * a.ff, a.ff, lane));
    }
    if (lane == 0) {
        if (a.accumulate) a.y32[(size_t)t * a.width + n] += acc;
        else a.y32[(size_t)t * a.width + n] = acc;
    }
}

// ------------------------------------------------------------------------------------------------ several tokens: expert by expert (bf16)
// 16 weight rows are the M side of m16n8k16 tiles, the tokens that chose the expert the N side (NB times 8); the CTA's warps split K.  The order of
// the 32 k of a step is permuted alike for both operands, which a dot product does not notice: 16-byte loads everywhere.
constexpr int MG_WARPS = 8, MG_MAX_T = 16;

// one step of 32 k: rows wa, wb (16 bytes per lane) and NB tokens' activations
template <int NB>
__device__ __forceinline__ void moe_mma_step(float (*c)[4], const bf16* wa, const bf16* wb, const bf16* const* x, int k, int K) {
    uint4 va = make_uint4(0, 0, 0, 0), vb = va, vx[NB];
#pragma unroll
    for (int i = 0; i < NB; ++i) vx[i] = make_uint4(0, 0, 0, 0);
    if (k < K) {
        va = *reinterpret_cast<const uint4*>(wa + k);
        vb = *reinterpret_cast<const uint4*>(wb + k);
#pragma unroll
        for (int i = 0; i < NB; ++i)
            if (x[i]) vx[i] = *reinterpret_cast<const uint4*>(x[i] + k);
    }
    const uint32_t a0[4] = {va.x, vb.x, va.y, vb.y}, a1[4] = {va.z, vb.z, va.w, vb.w};
#pragma unroll
    for (int i = 0; i < NB; ++i) {
        mma_bf16(c[i], a0, vx[i].x, vx[i].y);
        mma_bf16(c[i], a1, vx[i].z, vx[i].w);
    }
}

// grid (blocks of 16 weight rows, experts): 8 hidden units (gate and up rows interleaved) or 16 (glu 2) of one expert for all its tokens
template <int NB>
__global__ void __launch_bounds__(MG_WARPS * 32) moe_gateup_mma_kernel(MoeSparseArgs a, int T_) {
    __shared__ float part[MG_WARPS][16][8 * NB + 1];
    __shared__ int list[MG_MAX_T];  // slots (token * top + k) that chose this expert
    __shared__ int count;
    const int e = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
    if (warp == 0) {
        int n = 0;
        for (int s0 = 0; s0 < T_ * a.top; s0 += 32) {
            const bool hit = s0 + lane < T_ * a.top && a.idx[s0 + lane] == e;
            const unsigned mask = __ballot_sync(0xffffffffu, hit);
            const int at = n + __popc(mask & ((1u << lane) - 1u));
            if (hit && at < MG_MAX_T) list[at] = s0 + lane;
            n += __popc(mask);
        }
        if (lane == 0) count = min(n, MG_MAX_T);
    }
    __syncthreads();
    const int n_tok = count;
    if (n_tok == 0) return;
    const int rows = a.glu == 2 ? a.ff : 2 * a.ff, n0 = blockIdx.x * 16;
    const bf16* W = static_cast<const bf16*>(a.w13) + (size_t)e * rows * a.width;
    const bf16* wa = W + (size_t)min(n0 + gid, rows - 1) * a.width;
    const bf16* wb = W + (size_t)min(n0 + gid + 8, rows - 1) * a.width;
    const bf16* x[NB];
    float c[NB][4];
#pragma unroll
    for (int i = 0; i < NB; ++i) {
        x[i] = i * 8 + gid < n_tok ? static_cast<const bf16*>(a.h) + (size_t)(list[i * 8 + gid] / a.top) * a.width : nullptr;
        c[i][0] = c[i][1] = c[i][2] = c[i][3] = 0.f;
    }
#pragma unroll 4
    for (int kb = warp * 32; kb < a.width; kb += MG_WARPS * 32) moe_mma_step<NB>(c, wa, wb, x, kb + tig * 8, a.width);
#pragma unroll
    for (int i = 0; i < NB; ++i) {
        part[warp][gid][i * 8 + tig * 2] = c[i][0]; part[warp][gid][i * 8 + tig * 2 + 1] = c[i][1];
        part[warp][gid + 8][i * 8 + tig * 2] = c[i][2]; part[warp][gid + 8][i * 8 + tig * 2 + 1] = c[i][3];
    }
    __syncthreads();
    bf16* act = static_cast<bf16*>(a.act);
    for (int i = threadIdx.x; i < 8 * n_tok; i += blockDim.x) {
        const int m = i >> 3, r = (i & 7) * 2, n = n0 + r, slot = list[m];
        float g = 0.f, u = 0.f;
#pragma unroll
        for (int w = 0; w < MG_WARPS; ++w) { g += part[w][r][m]; u += part[w][r + 1][m]; }
        if (n >= rows) continue;
        g = rnd<bf16>(g); u = rnd<bf16>(u);
        if (a.glu == 2) {
            g = fmaxf(g, 0.f); u = fmaxf(u, 0.f);
            act[(size_t)slot * a.ff + n] = from_f<bf16>(g * g);
            if (n + 1 < rows) act[(size_t)slot * a.ff + n + 1] = from_f<bf16>(u * u);
        } else if (a.glu == 1) {
            const float w = a.wsel[slot];
            g = fminf(g * w, a.limit);
            u = fminf(fmaxf(u * w, -a.limit), a.limit);
            act[(size_t)slot * a.ff + (n >> 1)] = from_f<bf16>(g * sigmoid_exact(a.alpha * g) * (u + 1.f));
        } else {
            act[(size_t)slot * a.ff + (n >> 1)] = from_f<bf16>(g * sigmoid_exact(g) * u);
        }
    }
}

// grid (blocks of 16 output columns): the experts one after the other, every expert's product weighted per token in fp32.
// dynamic shared memory: slot of (expert, token) [E][T] (-1: not chosen), then one flag per expert
template <int NB>
__global__ void __launch_bounds__(2 * MG_WARPS * 32) moe_down_mma_kernel(MoeSparseArgs a, int T_) {
    constexpr int NW = 2 * MG_WARPS;
    extern __shared__ int slot_of[];
    int* used = slot_of + a.E * T_;
    __shared__ float part[NW][16][8 * NB + 1];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3, n0 = blockIdx.x * 16;
    for (int i = threadIdx.x; i < a.E * T_ + a.E; i += blockDim.x) slot_of[i] = i < a.E * T_ ? -1 : 0;
    __syncthreads();
    for (int s = threadIdx.x; s < T_ * a.top; s += blockDim.x) {
        const int e = a.idx[s];
        if (e < a.E) { slot_of[e * T_ + s / a.top] = s; used[e] = 1; }
    }
    __syncthreads();
    const bf16* W = static_cast<const bf16*>(a.w2);
    const bf16* wa = W + (size_t)min(n0 + gid, a.width - 1) * a.E * a.ff;
    const bf16* wb = W + (size_t)min(n0 + gid + 8, a.width - 1) * a.E * a.ff;
    float sum[NB][4];
#pragma unroll
    for (int i = 0; i < NB; ++i) sum[i][0] = sum[i][1] = sum[i][2] = sum[i][3] = 0.f;
    for (int e = 0; e < a.E; ++e) {
        if (!used[e]) continue;
        const bf16* x[NB];
        float c[NB][4];
#pragma unroll
        for (int i = 0; i < NB; ++i) {
            const int t = i * 8 + gid, s = t < T_ ? slot_of[e * T_ + t] : -1;
            x[i] = s >= 0 ? static_cast<const bf16*>(a.act) + (size_t)s * a.ff : nullptr;
            c[i][0] = c[i][1] = c[i][2] = c[i][3] = 0.f;
        }
#pragma unroll 4
        for (int kb = warp * 32; kb < a.ff; kb += NW * 32) moe_mma_step<NB>(c, wa + (size_t)e * a.ff, wb + (size_t)e * a.ff, x, kb + tig * 8, a.ff);
#pragma unroll
        for (int i = 0; i < NB; ++i) {
            float w[2];
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int t = i * 8 + tig * 2 + u, s = t < T_ ? slot_of[e * T_ + t] : -1;
                w[u] = s < 0 ? 0.f : a.glu == 1 ? 1.f : a.wsel[s];
            }
            sum[i][0] = fmaf(w[0], c[i][0], sum[i][0]); sum[i][1] = fmaf(w[1], c[i][1], sum[i][1]);
            sum[i][2] = fmaf(w[0], c[i][2], sum[i][2]); sum[i][3] = fmaf(w[1], c[i][3], sum[i][3]);
        }
    }
#pragma unroll
    for (int i = 0; i < NB; ++i) {
        part[warp][gid][i * 8 + tig * 2] = sum[i][0]; part[warp][gid][i * 8 + tig * 2 + 1] = sum[i][1];
        part[warp][gid + 8][i * 8 + tig * 2] = sum[i][2]; part[warp][gid + 8][i * 8 + tig * 2 + 1] = sum[i][3];
    }
    __syncthreads();
    for (int i = threadIdx.x; i < 16 * T_; i += blockDim.x) {
        const int t = i >> 4, r = i & 15, n = n0 + r;
        if (n >= a.width) continue;
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < NW; ++w) v += part[w][r][t];
        for (int k = 0; k < a.top; ++k)  // identity experts
            if (a.idx[t * a.top + k] >= a.E) v += a.wsel[t * a.top + k] * to_f(static_cast<const bf16*>(a.h)[(size_t)t * a.width + n]);
        float* y = a.y32 + (size_t)t * a.width + n;
        *y = a.accumulate ? *y + v : v;
    }
}

template <int NB> inline void run_moe_mma(const MoeSparseArgs& a, int T_, cudaStream_t st) {
    const int rows = a.glu == 2 ? a.ff : 2 * a.ff;
    moe_gateup_mma_kernel<NB><<<dim3((unsigned)((rows + 15) / 16), (unsigned)a.E), MG_WARPS * 32, 0, st>>>(a, T_);
    moe_down_mma_kernel<NB><<<(unsigned)((a.width + 15) / 16), 2 * MG_WARPS * 32, sizeof(int) * (size_t)a.E * (T_ + 1), st>>>(a, T_);
}
// true when the shapes suit the two kernels above; launches them
inline bool launch_moe_mma(const MoeSparseArgs& a, int64_t T_, cudaStream_t st) {
    if (T_ < 2 || T_ > MG_MAX_T || a.width % 8 || a.ff % 8 || a.E > 400) return false;
    if ((reinterpret_cast<uintptr_t>(a.h) | reinterpret_cast<uintptr_t>(a.w13) | reinterpret_cast<uintptr_t>(a.w2) | reinterpret_cast<uintptr_t>(a.act)) % 16) return false;
    if (T_ <= 8) run_moe_mma<1>(a, (int)T_, st);
    else run_moe_mma<2>(a, (int)T_, st);
    return true;
}

// y[t, :] += (sum of dense[t, first .. n - 1]) * h[t, :]
template <typename T>
__global__ void rows_axpy_kernel(float* __restrict__ y, const T* __restrict__ h, const float* __restrict__ dense, int n, int first, int D) {
    const int t = blockIdx.x;
    float w = 0.f;
    for (int e = first; e < n; ++e) w += dense[(size_t)t * n + e];
    if (w == 0.f) return;
    for (int i = threadIdx.x; i < D; i += blockDim.x) y[(size_t)t * D + i] += w * to_f(h[(size_t)t * D + i]);
}

}  // namespace mbh
