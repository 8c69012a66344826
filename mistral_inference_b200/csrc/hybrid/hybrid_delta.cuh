// Gated delta rule: linear attention whose state forgets per key channel and writes only what it does not already predict.
//
//     S <- diag(g_t) S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t         per head, S [d, e] fp32, in the cache
//
// q, k and v are projections that went through a short causal convolution over time (per channel, last tap = the current token) and
// SiLU; q and k are unit vectors per head (q also times d^(-1/2)); beta = sigmoid of a projection; g = exp(-exp(A_log_h) softplus(z)) per head
// and key channel, z a low-rank projection plus a bias (written by the decay epilogue of the Linear that makes z).
//
//   delta_prep       prompts: convolution, SiLU, unit norms, k . q, beta of every token, from the packed projection
//   delta_conv_state the last inputs of the convolutions of each sequence -> the cache
//   delta_scan       the recurrence over a whole prompt (portion)
//   delta_step       one token per sequence: everything between the input projection and the output projection in one launch
//
// Reading out after the write, o = S_new^T q = S_old^T (g q) + u (k . q), and u needs S_old^T (g k): both sums run over the OLD state side
// by side, so a token costs one reduction, not two in a row.  A state column is spread over LANES lanes of a warp (LANES * RPL4 * 4 >= d
// rows, four neighbouring rows per lane and step, so shared and global memory are read 16 bytes at a time without bank conflicts); columns
// are independent.  The state is kept column by column, [slots, H, e, d].
//
// The convolution's inputs of a sequence are a ring of `taps` rows, input at position p in row p % taps: a decode step writes the row that no
// CTA of the same launch reads (position p - taps), so heads that share a key head need no order among them.
#pragma once
#include "hybrid_common.cuh"

namespace mbh {

struct DeltaArgs {
    const void* y;          // [T, y_pitch] projections: q (G*d) | k (G*d) | v (H*e) | beta logits (H) | decay latent (ra) | gate latent (rg) | ...
    int y_pitch, ra, rg;
    const void* conv;       // [2*G*d + H*e, taps]
    int taps;
    float* cstate;          // [slots, taps, 2*G*d + H*e] last inputs of the convolutions
    float* state;           // [slots, H, e, d]
    const int* positions;   // [T]
    const int* q_start;     // [B + 1]
    const int* seqpos;      // [B] tokens before this call
    const int* slots;       // [B]
    int T, B, H, G, d, e;
    // prompts
    float* qk;              // [T, 2, G*d] unit vectors (q scaled)
    float* kq;              // [T, G] k . q
    float* v;               // [T, H*e]
    float* beta;            // [T, H]
    const float* g;         // [T, H*d] decays
    float* o;               // [T, H*e]
    // decode step
    const void* w_a2; const void* dt_bias; const void* a_log;   // [H*d, ra], [H*d], [H]
    const void* w_g2; const void* norm;                         // [H*e, rg], [e]
    float eps;
    void* out;              // [B, H*e]
};

__device__ __forceinline__ float delta_decay(float z, float a_log) { return expf(-expf(a_log) * softplus_exact(z)); }
__device__ __forceinline__ float silu_exact(float x) { return x * sigmoid_exact(x); }

constexpr float DELTA_UNIT_EPS = 1e-6f;

// convolution of channel ch at token t (place i of its sequence in this call, absolute position pos), before the SiLU
template <typename T>
__device__ __forceinline__ float delta_conv(const DeltaArgs& a, int t, int i, int pos, const float* cs, int channels, int ch) {
    const T* w = static_cast<const T*>(a.conv) + (size_t)ch * a.taps;
    const T* col = static_cast<const T*>(a.y) + (size_t)t * a.y_pitch + ch;
    float acc = 0.f;
    for (int j = 0; j < a.taps; ++j) {
        const int back = a.taps - 1 - j;
        float x = 0.f;
        if (back <= i) x = to_f(col[-(ptrdiff_t)back * a.y_pitch]);
        else if (back <= pos) x = cs[(size_t)((pos - back) % a.taps) * channels + ch];
        acc = fmaf(to_f(w[j]), x, acc);
    }
    return acc;
}

constexpr int DP_WARPS = 8;

// A warp per (token, unit): units 0 .. G-1 are the query and key vector of key head u, the next H the value heads.  The warps of a CTA take
// neighbouring tokens of the same unit (their convolution windows overlap).  NJ: channels per lane, d <= 32 * NJ.
template <typename T, int NJ>
__global__ void __launch_bounds__(DP_WARPS * 32) delta_prep_kernel(DeltaArgs a) {
    const int t = blockIdx.x * DP_WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (t >= a.T) return;
    int b = 0;
    while (b + 1 < a.B && a.q_start[b + 1] <= t) ++b;
    const int i = t - a.q_start[b], pos = a.positions[t], Nk = a.G * a.d, channels = 2 * Nk + a.H * a.e;
    const float* cs = a.cstate + (size_t)a.slots[b] * a.taps * channels;
    for (int u = blockIdx.y; u < a.G + a.H; u += gridDim.y) {
        if (u < a.G) {
            float q[NJ], k[NJ], qq = 0.f, kk = 0.f, kq = 0.f;
#pragma unroll
            for (int j = 0; j < NJ; ++j) {
                const int c = lane + 32 * j;
                q[j] = k[j] = 0.f;
                if (c < a.d) {
                    q[j] = silu_exact(delta_conv<T>(a, t, i, pos, cs, channels, u * a.d + c));
                    k[j] = silu_exact(delta_conv<T>(a, t, i, pos, cs, channels, Nk + u * a.d + c));
                }
                qq = fmaf(q[j], q[j], qq);
                kk = fmaf(k[j], k[j], kk);
            }
            const float iq = 1.f / (sqrtf(warp_sum(qq) + DELTA_UNIT_EPS) * sqrtf((float)a.d)), ik = 1.f / sqrtf(warp_sum(kk) + DELTA_UNIT_EPS);
            float* dst = a.qk + (size_t)t * 2 * Nk + u * a.d;
#pragma unroll
            for (int j = 0; j < NJ; ++j) {
                const int c = lane + 32 * j;
                q[j] *= iq; k[j] *= ik;
                kq = fmaf(k[j], q[j], kq);
                if (c < a.d) { dst[c] = q[j]; dst[Nk + c] = k[j]; }
            }
            kq = warp_sum(kq);
            if (lane == 0) a.kq[(size_t)t * a.G + u] = kq;
        } else {
            const int h = u - a.G;
            for (int c = lane; c < a.e; c += 32)
                a.v[(size_t)t * a.H * a.e + h * a.e + c] = silu_exact(delta_conv<T>(a, t, i, pos, cs, channels, 2 * Nk + h * a.e + c));
            if (lane == 0) a.beta[(size_t)t * a.H + h] = sigmoid_exact(to_f(static_cast<const T*>(a.y)[(size_t)t * a.y_pitch + channels + h]));
        }
    }
}

// grid (B, blocks of channels): the last taps - 1 inputs of each sequence of this call
template <typename T>
__global__ void delta_conv_state_kernel(DeltaArgs a) {
    const int b = blockIdx.x, channels = 2 * a.G * a.d + a.H * a.e, t1 = a.q_start[b + 1], len = t1 - a.q_start[b];
    float* cs = a.cstate + (size_t)a.slots[b] * a.taps * channels;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < channels; c += gridDim.y * blockDim.x)
        for (int back = min(a.taps - 1, len); back >= 1; --back)
            cs[(size_t)((a.seqpos[b] + len - back) % a.taps) * channels + c] = to_f(static_cast<const T*>(a.y)[(size_t)(t1 - back) * a.y_pitch + c]);
}

// LANES lanes hold a state column, RPL4 float4 each
template <int LANES, int RPL4> struct DeltaColumn {
    static constexpr int DMAX = LANES * RPL4 * 4;
    static __device__ __forceinline__ void load(const float* col, int d, int l, float (*S)[4]) {
#pragma unroll
        for (int j = 0; j < RPL4; ++j) {
            const int i = (j * LANES + l) * 4;
            if (d % 4 == 0) {
                const float4 v = i < d ? *reinterpret_cast<const float4*>(col + i) : make_float4(0.f, 0.f, 0.f, 0.f);
                S[j][0] = v.x; S[j][1] = v.y; S[j][2] = v.z; S[j][3] = v.w;
            } else {
#pragma unroll
                for (int u = 0; u < 4; ++u) S[j][u] = i + u < d ? col[i + u] : 0.f;
            }
        }
    }
    static __device__ __forceinline__ void store(float* col, int d, int l, const float (*S)[4]) {
#pragma unroll
        for (int j = 0; j < RPL4; ++j) {
            const int i = (j * LANES + l) * 4;
            if (d % 4 == 0) {
                if (i < d) *reinterpret_cast<float4*>(col + i) = make_float4(S[j][0], S[j][1], S[j][2], S[j][3]);
            } else {
#pragma unroll
                for (int u = 0; u < 4; ++u)
                    if (i + u < d) col[i + u] = S[j][u];
            }
        }
    }
    // one token: returns the read-out (the same in every lane of the column) and updates S.  gs / ks / gk / gq: [DMAX] shared memory,
    // zero beyond d
    static __device__ __forceinline__ float token(const float* gs, const float* ks, const float* gk, const float* gq, float kq, float v, float beta, int l,
                                                  float (*S)[4]) {
        float p0 = 0.f, p1 = 0.f, r0 = 0.f, r1 = 0.f;
#pragma unroll
        for (int j = 0; j < RPL4; ++j) {
            const int i = (j * LANES + l) * 4;
            const float4 a4 = *reinterpret_cast<const float4*>(gk + i), b4 = *reinterpret_cast<const float4*>(gq + i);
            p0 = fmaf(S[j][0], a4.x, p0); p1 = fmaf(S[j][1], a4.y, p1); p0 = fmaf(S[j][2], a4.z, p0); p1 = fmaf(S[j][3], a4.w, p1);
            r0 = fmaf(S[j][0], b4.x, r0); r1 = fmaf(S[j][1], b4.y, r1); r0 = fmaf(S[j][2], b4.z, r0); r1 = fmaf(S[j][3], b4.w, r1);
        }
        float p = p0 + p1, r = r0 + r1;
#pragma unroll
        for (int o = LANES / 2; o > 0; o >>= 1) {
            p += __shfl_xor_sync(0xffffffffu, p, o);
            r += __shfl_xor_sync(0xffffffffu, r, o);
        }
        const float u = beta * (v - p);
#pragma unroll
        for (int j = 0; j < RPL4; ++j) {
            const int i = (j * LANES + l) * 4;
            const float4 g4 = *reinterpret_cast<const float4*>(gs + i), k4 = *reinterpret_cast<const float4*>(ks + i);
            S[j][0] = fmaf(k4.x, u, g4.x * S[j][0]); S[j][1] = fmaf(k4.y, u, g4.y * S[j][1]);
            S[j][2] = fmaf(k4.z, u, g4.z * S[j][2]); S[j][3] = fmaf(k4.w, u, g4.w * S[j][3]);
        }
        return fmaf(u, kq, r);
    }
};

constexpr int DS_THREADS = 128;

// One CTA per (sequence, head, block of DS_THREADS / LANES columns).  TB tokens at a time go through shared memory, the next tile is fetched
// into registers meanwhile.
template <int LANES, int RPL4, int TB>
__global__ void __launch_bounds__(DS_THREADS) delta_scan_kernel(DeltaArgs a) {
    using Col = DeltaColumn<LANES, RPL4>;
    constexpr int D = Col::DMAX, R = TB * D / DS_THREADS, COLS = DS_THREADS / LANES;
    static_assert(TB * D % DS_THREADS == 0 && TB * COLS <= 4 * DS_THREADS, "tile shape");
    __shared__ __align__(16) float gs[TB][D], ks[TB][D], gk[TB][D], gq[TB][D];
    __shared__ float vs[TB][COLS], os[TB][COLS], bs[TB], kqs[TB];
    const int b = blockIdx.x / a.H, h = blockIdx.x % a.H, kvh = h / (a.H / a.G);
    const int l = threadIdx.x % LANES, cl = threadIdx.x / LANES, c0 = blockIdx.y * COLS, c = c0 + cl;
    const int t0 = a.q_start[b], t1 = a.q_start[b + 1], Nk = a.G * a.d, Hd = a.H * a.d, He = a.H * a.e;
    if (t0 >= t1) return;
    float* col = a.state + (((size_t)a.slots[b] * a.H + h) * a.e + min(c, a.e - 1)) * a.d;
    float S[RPL4][4];
    if (a.seqpos[b] > 0) {
        Col::load(col, a.d, l, S);
    } else {
#pragma unroll
        for (int j = 0; j < RPL4; ++j) S[j][0] = S[j][1] = S[j][2] = S[j][3] = 0.f;
    }
    float pq[R], pk[R], pg[R], pv[(TB * COLS + DS_THREADS - 1) / DS_THREADS], pb = 0.f, pkq = 0.f;
    constexpr int RV = (TB * COLS + DS_THREADS - 1) / DS_THREADS;
    auto fetch = [&](int tb) {
#pragma unroll
        for (int r = 0; r < R; ++r) {
            const int idx = threadIdx.x + r * DS_THREADS, tt = idx / D, i = idx % D;
            const bool ok = tb + tt < t1 && i < a.d;
            const float* src = a.qk + (size_t)(tb + tt) * 2 * Nk + kvh * a.d + i;
            pq[r] = ok ? src[0] : 0.f;
            pk[r] = ok ? src[Nk] : 0.f;
            pg[r] = ok ? a.g[(size_t)(tb + tt) * Hd + h * a.d + i] : 0.f;
        }
#pragma unroll
        for (int r = 0; r < RV; ++r) {
            const int idx = threadIdx.x + r * DS_THREADS, tt = idx / COLS, cc = c0 + idx % COLS;
            pv[r] = (tt < TB && tb + tt < t1 && cc < a.e) ? a.v[(size_t)(tb + tt) * He + h * a.e + cc] : 0.f;
        }
        if (threadIdx.x < TB && tb + (int)threadIdx.x < t1) {
            pb = a.beta[(size_t)(tb + threadIdx.x) * a.H + h];
            pkq = a.kq[(size_t)(tb + threadIdx.x) * a.G + kvh];
        }
    };
    fetch(t0);
    for (int tb = t0; tb < t1; tb += TB) {
        const int nt = min(TB, t1 - tb);
        __syncthreads();
#pragma unroll
        for (int r = 0; r < R; ++r) {
            const int idx = threadIdx.x + r * DS_THREADS, tt = idx / D, i = idx % D;
            gs[tt][i] = pg[r]; ks[tt][i] = pk[r]; gk[tt][i] = pg[r] * pk[r]; gq[tt][i] = pg[r] * pq[r];
        }
#pragma unroll
        for (int r = 0; r < RV; ++r) {
            const int idx = threadIdx.x + r * DS_THREADS;
            if (idx < TB * COLS) vs[idx / COLS][idx % COLS] = pv[r];
        }
        if (threadIdx.x < TB) { bs[threadIdx.x] = pb; kqs[threadIdx.x] = pkq; }
        __syncthreads();
        if (tb + TB < t1) fetch(tb + TB);
        for (int tt = 0; tt < nt; ++tt) {
            const float o = Col::token(gs[tt], ks[tt], gk[tt], gq[tt], kqs[tt], vs[tt][cl], bs[tt], l, S);
            if (l == 0) os[tt][cl] = o;
        }
        __syncthreads();
#pragma unroll
        for (int r = 0; r < RV; ++r) {
            const int idx = threadIdx.x + r * DS_THREADS, tt = idx / COLS, cc = c0 + idx % COLS;
            if (tt < nt && cc < a.e) a.o[(size_t)(tb + tt) * He + h * a.e + cc] = os[tt][idx % COLS];
        }
    }
    if (c < a.e) Col::store(col, a.d, l, S);
}

// dot product of two rows of K elements over 8 neighbouring lanes (x in shared memory); every lane of the eight gets the sum
template <typename T>
__device__ __forceinline__ float dot8(const T* __restrict__ w, const float* x, int K, int l8) {
    constexpr int V = Vec<T>::N;
    float acc = 0.f;
    if (K % V == 0 && reinterpret_cast<uintptr_t>(w) % 16 == 0) {
        for (int k = l8 * V; k < K; k += 8 * V) {
            float wv[V];
            Vec<T>::load(w + k, wv);
#pragma unroll
            for (int i = 0; i < V; ++i) acc = fmaf(wv[i], x[k + i], acc);
        }
    } else {
        for (int k = l8; k < K; k += 8) acc = fmaf(to_f(w[k]), x[k], acc);
    }
    acc += __shfl_xor_sync(0xffffffffu, acc, 1);
    acc += __shfl_xor_sync(0xffffffffu, acc, 2);
    return acc + __shfl_xor_sync(0xffffffffu, acc, 4);
}

constexpr int DT_THREADS = 512, DT_PASS = 2;

// One CTA per (sequence, head), one token: convolutions and unit norms, decays (second half of their low-rank projection included), beta, the
// state update and read-out, the head's norm, and the output gate (second half of its projection included).  Shared memory:
// qs ks gs gk gq [DMAX] | v gate o [e] | decay latent [ra] | gate latent [rg]
template <typename T, int LANES, int RPL4>
__global__ void __launch_bounds__(DT_THREADS) delta_step_kernel(DeltaArgs a) {
    using Col = DeltaColumn<LANES, RPL4>;
    constexpr int D = Col::DMAX, COLS = DT_THREADS / LANES;
    extern __shared__ __align__(16) float dsm[];
    float *qs = dsm, *ks = qs + D, *gs = ks + D, *gk = gs + D, *gq = gk + D, *vs = gq + D, *gate = vs + a.e, *os = gate + a.e, *la = os + a.e, *lg = la + a.ra;
    __shared__ float red[32], sc[3];
    const int b = blockIdx.x / a.H, h = blockIdx.x % a.H, rep = a.H / a.G, kvh = h / rep, tid = threadIdx.x;
    const int Nk = a.G * a.d, channels = 2 * Nk + a.H * a.e, pos = a.positions[b], slot = a.slots[b];
    const int l = tid % LANES, cl = tid / LANES;
    float* heads = a.state + ((size_t)slot * a.H + h) * a.e * a.d;
    // the state of the first columns is on its way while the inputs are prepared
    float S[DT_PASS][RPL4][4];
    const bool old = a.seqpos[b] > 0;
#pragma unroll
    for (int p = 0; p < DT_PASS; ++p) {
        const int c = p * COLS + cl;
        if (old && c < a.e) Col::load(heads + (size_t)c * a.d, a.d, l, S[p]);
        else {
#pragma unroll
            for (int j = 0; j < RPL4; ++j) S[p][j][0] = S[p][j][1] = S[p][j][2] = S[p][j][3] = 0.f;
        }
    }
    const T* row = static_cast<const T*>(a.y) + (size_t)b * a.y_pitch;
    for (int i = tid; i < a.ra; i += DT_THREADS) la[i] = to_f(row[channels + a.H + i]);
    for (int i = tid; i < a.rg; i += DT_THREADS) lg[i] = to_f(row[channels + a.H + a.ra + i]);
    float* cs = a.cstate + (size_t)slot * a.taps * channels;
    for (int i = tid; i < 2 * D + a.e; i += DT_THREADS) {
        const int which = i < D ? 0 : i < 2 * D ? 1 : 2, c = i - min(which, 2) * D;
        if (which < 2 && c >= a.d) { (which ? ks : qs)[c] = 0.f; continue; }
        const int ch = which == 0 ? kvh * a.d + c : which == 1 ? Nk + kvh * a.d + c : 2 * Nk + h * a.e + c;
        const float x = silu_exact(delta_conv<T>(a, b, 0, pos, cs, channels, ch));
        (which == 0 ? qs : which == 1 ? ks : vs)[c] = x;
        if (a.taps > 1 && (which == 2 || h % rep == 0)) cs[(size_t)(pos % a.taps) * channels + ch] = to_f(row[ch]);
    }
    __syncthreads();
    const int warp = tid >> 5, lane = tid & 31;
    if (warp < 2) {  // squared lengths of q and k
        const float* x = warp ? ks : qs;
        float ss = 0.f;
        for (int i = lane; i < a.d; i += 32) ss = fmaf(x[i], x[i], ss);
        ss = warp_sum(ss);
        if (lane == 0) sc[warp] = warp ? 1.f / sqrtf(ss + DELTA_UNIT_EPS) : 1.f / (sqrtf(ss + DELTA_UNIT_EPS) * sqrtf((float)a.d));
    } else if (warp == 2) {
        float dq = 0.f;
        for (int i = lane; i < a.d; i += 32) dq = fmaf(ks[i], qs[i], dq);
        dq = warp_sum(dq);
        if (lane == 0) sc[2] = dq;
    }
    {   // decays and gate logits: eight lanes per row of the second projections
        const float alog = to_f(static_cast<const T*>(a.a_log)[h]);
        for (int r0 = 0; r0 < a.d + a.e; r0 += DT_THREADS / 8) {
            const int r = r0 + (tid >> 3), l8 = tid & 7;
            const bool is_d = r < a.d, live = r < a.d + a.e;
            const int rr = live ? (is_d ? h * a.d + r : h * a.e + r - a.d) : 0;
            const T* w = is_d ? static_cast<const T*>(a.w_a2) + (size_t)rr * a.ra : static_cast<const T*>(a.w_g2) + (size_t)rr * a.rg;
            const float s = dot8<T>(w, is_d ? la : lg, is_d ? a.ra : a.rg, l8);
            if (live && l8 == 0) {
                if (is_d) gs[r] = delta_decay(s + to_f(static_cast<const T*>(a.dt_bias)[rr]), alog);
                else gate[r - a.d] = sigmoid_exact(rnd<T>(s));
            }
        }
        for (int i = a.d + tid; i < D; i += DT_THREADS) gs[i] = 0.f;
    }
    __syncthreads();
    const float iq = sc[0], ik = sc[1], kq = sc[2] * iq * ik;
    for (int i = tid; i < D; i += DT_THREADS) {
        const float k = ks[i] * ik;
        ks[i] = k;
        gk[i] = gs[i] * k;
        gq[i] = gs[i] * (qs[i] * iq);
    }
    __syncthreads();
    const float beta = sigmoid_exact(to_f(row[channels + h]));
    for (int c0 = 0; c0 < a.e; c0 += DT_PASS * COLS) {
#pragma unroll
        for (int p = 0; p < DT_PASS; ++p) {
            const int c = c0 + p * COLS + cl;
            if (c0 > 0) {
                if (old && c < a.e) Col::load(heads + (size_t)c * a.d, a.d, l, S[p]);
                else {
#pragma unroll
                    for (int j = 0; j < RPL4; ++j) S[p][j][0] = S[p][j][1] = S[p][j][2] = S[p][j][3] = 0.f;
                }
            }
            const float o = Col::token(gs, ks, gk, gq, kq, c < a.e ? vs[c] : 0.f, beta, l, S[p]);
            if (c < a.e) {
                if (l == 0) os[c] = o;
                Col::store(heads + (size_t)c * a.d, a.d, l, S[p]);
            }
        }
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = tid; c < a.e; c += DT_THREADS) ss = fmaf(os[c], os[c], ss);
    ss = block_sum(ss, red);
    const float inv = 1.f / sqrtf(ss / (float)a.e + a.eps);
    T* out = static_cast<T*>(a.out) + (size_t)b * a.H * a.e + h * a.e;
    for (int c = tid; c < a.e; c += DT_THREADS) out[c] = from_f<T>(os[c] * inv * to_f(static_cast<const T*>(a.norm)[c]) * gate[c]);
}

}  // namespace mbh
