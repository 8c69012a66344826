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
// Reading out after the write, o = S_new^T q = (g S_old)^T q + u (k . q), and u needs (g S_old)^T k: both sums run over the decayed OLD state
// side by side, so a token costs one reduction, not two in a row.  A state column is spread over LANES lanes of a warp (LANES * RPL4 * 4 >= d
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
    int stage;              // the second projections' slices of a head go through shared memory
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

// The same for the usual sizes (taps <= 4, channel counts and addresses that allow four channels at a time): a warp takes one unit of DP_TILE
// consecutive tokens and walks them with the convolution's reach in registers, so every projection is read once (plus the reach where a tile or
// a sequence starts).  A lane owns four neighbouring channels of each block of 128; NB blocks cover a head's key channels, d <= 128 * NB.
// The inputs of DP_AHEAD tokens are loaded before the first of them is used.
constexpr int DP_TILE = 16, DP_AHEAD = 4;

template <typename T, int TAPS>
struct DeltaConvWalk {
    float w[4][TAPS], win[TAPS > 1 ? TAPS - 1 : 1][4];
    __device__ __forceinline__ void weights(const T* conv, int ch) {
        float f[4 * TAPS];  // the four channels' taps follow one another
#pragma unroll
        for (int j = 0; j < TAPS; ++j) load4(conv + (size_t)ch * TAPS + 4 * j, f + 4 * j);
#pragma unroll
        for (int i = 0; i < 4 * TAPS; ++i) w[i / TAPS][i % TAPS] = f[i];
    }
    // inputs of the TAPS - 1 tokens before token t (place i of its sequence, position pos); col: &y[t][ch], cs: the carried inputs
    __device__ __forceinline__ void reach(const T* col, int pitch, int i, int pos, const float* cs, int channels, int ch) {
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) {
            const int back = TAPS - 1 - j;
            if (back <= i) load4(col - (ptrdiff_t)back * pitch, win[j]);
            else if (back <= pos) load4(cs + (size_t)((pos - back) % TAPS) * channels + ch, win[j]);
            else win[j][0] = win[j][1] = win[j][2] = win[j][3] = 0.f;
        }
    }
    __device__ __forceinline__ void step(const float* x, float* out) {
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            float acc = w[u][TAPS - 1] * x[u];
#pragma unroll
            for (int j = 0; j < TAPS - 1; ++j) acc = fmaf(w[u][j], win[j][u], acc);
            // bf16 storage: fast exponential and division (relative error about 1e-6, far below the storage type of the inputs)
            out[u] = sizeof(T) == 2 ? __fdividef(acc, 1.f + __expf(-acc)) : silu_exact(acc);
#pragma unroll
            for (int j = 0; j + 1 < TAPS - 1; ++j) win[j][u] = win[j + 1][u];
            if (TAPS > 1) win[TAPS > 1 ? TAPS - 2 : 0][u] = x[u];
        }
    }
};

template <typename T, int TAPS, int NB>
__global__ void __launch_bounds__(DP_WARPS * 32) delta_prep_tiled_kernel(DeltaArgs a) {
    const int lane = threadIdx.x & 31, t0 = (blockIdx.x * DP_WARPS + (threadIdx.x >> 5)) * DP_TILE, t1 = min(t0 + DP_TILE, a.T);
    if (t0 >= a.T) return;
    const int Nk = a.G * a.d, channels = 2 * Nk + a.H * a.e, u = blockIdx.y;
    const T* conv = static_cast<const T*>(a.conv);
    const T* Y = static_cast<const T*>(a.y);
    int b = 0;
    while (b + 1 < a.B && a.q_start[b + 1] <= t0) ++b;
    int seq_end = t0;  // forces the reach to be loaded at the first token
    if (u < a.G) {
        DeltaConvWalk<T, TAPS> Q[NB], K[NB];
#pragma unroll
        for (int n = 0; n < NB; ++n) {
            const int c = n * 128 + lane * 4;
            if (c < a.d) { Q[n].weights(conv, u * a.d + c); K[n].weights(conv, Nk + u * a.d + c); }
        }
        for (int tb = t0; tb < t1; tb += DP_AHEAD) {
          float xq[DP_AHEAD][NB][4], xk[DP_AHEAD][NB][4];
#pragma unroll
          for (int s = 0; s < DP_AHEAD; ++s) {
            const T* row = Y + (size_t)min(tb + s, t1 - 1) * a.y_pitch + u * a.d;
#pragma unroll
            for (int n = 0; n < NB; ++n) {
                const int c = n * 128 + lane * 4;
                if (c < a.d) { load4(row + c, xq[s][n]); load4(row + Nk + c, xk[s][n]); }
            }
          }
#pragma unroll
          for (int s = 0; s < DP_AHEAD; ++s) {
            const int t = tb + s;
            if (t >= t1) break;
            const T* row = Y + (size_t)t * a.y_pitch + u * a.d;
            if (t >= seq_end) {
                while (b + 1 < a.B && a.q_start[b + 1] <= t) ++b;
                seq_end = a.q_start[b + 1];
                const float* cs = a.cstate + (size_t)a.slots[b] * a.taps * channels;
                const int i = t - a.q_start[b], pos = a.positions[t];
#pragma unroll
                for (int n = 0; n < NB; ++n) {
                    const int c = n * 128 + lane * 4;
                    if (c < a.d) {
                        Q[n].reach(row + c, a.y_pitch, i, pos, cs, channels, u * a.d + c);
                        K[n].reach(row + Nk + c, a.y_pitch, i, pos, cs, channels, Nk + u * a.d + c);
                    }
                }
            }
            float q[NB][4], k[NB][4], qq = 0.f, kk = 0.f, kq = 0.f;
#pragma unroll
            for (int n = 0; n < NB; ++n) {
                const int c = n * 128 + lane * 4;
                if (c < a.d) { Q[n].step(xq[s][n], q[n]); K[n].step(xk[s][n], k[n]); }
                else {
#pragma unroll
                    for (int x = 0; x < 4; ++x) q[n][x] = k[n][x] = 0.f;
                }
#pragma unroll
                for (int x = 0; x < 4; ++x) { qq = fmaf(q[n][x], q[n][x], qq); kk = fmaf(k[n][x], k[n][x], kk); kq = fmaf(k[n][x], q[n][x], kq); }
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) {
                qq += __shfl_xor_sync(0xffffffffu, qq, o);
                kk += __shfl_xor_sync(0xffffffffu, kk, o);
                kq += __shfl_xor_sync(0xffffffffu, kq, o);
            }
            const float iq = 1.f / (sqrtf(qq + DELTA_UNIT_EPS) * sqrtf((float)a.d)), ik = 1.f / sqrtf(kk + DELTA_UNIT_EPS);
            float* dst = a.qk + (size_t)t * 2 * Nk + u * a.d;
#pragma unroll
            for (int n = 0; n < NB; ++n) {
                const int c = n * 128 + lane * 4;
                if (c < a.d) {
#pragma unroll
                    for (int x = 0; x < 4; ++x) { q[n][x] *= iq; k[n][x] *= ik; }
                    store4<float>(dst + c, q[n]);
                    store4<float>(dst + Nk + c, k[n]);
                }
            }
            if (lane == 0) a.kq[(size_t)t * a.G + u] = kq * iq * ik;
          }
        }
        return;
    }
    const int h = u - a.G;
    for (int c = lane * 4; c < a.e; c += 128) {
        const int ch = 2 * Nk + h * a.e + c;
        DeltaConvWalk<T, TAPS> V;
        V.weights(conv, ch);
        int bb = b;
        seq_end = t0;
        for (int tb = t0; tb < t1; tb += DP_AHEAD) {
          float x[DP_AHEAD][4];
#pragma unroll
          for (int s = 0; s < DP_AHEAD; ++s) load4(Y + (size_t)min(tb + s, t1 - 1) * a.y_pitch + ch, x[s]);
#pragma unroll
          for (int s = 0; s < DP_AHEAD; ++s) {
            const int t = tb + s;
            if (t >= t1) break;
            const T* col = Y + (size_t)t * a.y_pitch + ch;
            if (t >= seq_end) {
                while (bb + 1 < a.B && a.q_start[bb + 1] <= t) ++bb;
                seq_end = a.q_start[bb + 1];
                V.reach(col, a.y_pitch, t - a.q_start[bb], a.positions[t], a.cstate + (size_t)a.slots[bb] * a.taps * channels, channels, ch);
            }
            float v[4];
            V.step(x[s], v);
            store4<float>(a.v + (size_t)t * a.H * a.e + h * a.e + c, v);
          }
        }
    }
    for (int t = t0 + lane; t < t1; t += 32) a.beta[(size_t)t * a.H + h] = sigmoid_exact(to_f(Y[(size_t)t * a.y_pitch + channels + h]));
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
    static __device__ __forceinline__ void load(const float* col, int d, int l, float (&S)[RPL4][4]) {
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
    static __device__ __forceinline__ void store(float* col, int d, int l, const float (&S)[RPL4][4]) {
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
    // one token for C columns: o gets the read-outs (the same in every lane of a column), S the new state.  gs / ks / qs: [DMAX] shared memory,
    // zero beyond d; each value read serves C columns
    template <int C>
    static __device__ __forceinline__ void token(const float* gs, const float* ks, const float* qs, float kq, const float (&v)[C], float beta, int l,
                                                 float (&S)[C][RPL4][4], float (&o)[C]) {
        float4 k4[RPL4];
        float p[C][2], r[C][2];
#pragma unroll
        for (int c = 0; c < C; ++c) p[c][0] = p[c][1] = r[c][0] = r[c][1] = 0.f;
#pragma unroll
        for (int j = 0; j < RPL4; ++j) {
            const int i = (j * LANES + l) * 4;
            const float4 g4 = *reinterpret_cast<const float4*>(gs + i), q4 = *reinterpret_cast<const float4*>(qs + i);
            k4[j] = *reinterpret_cast<const float4*>(ks + i);
#pragma unroll
            for (int c = 0; c < C; ++c) {
                S[c][j][0] *= g4.x; S[c][j][1] *= g4.y; S[c][j][2] *= g4.z; S[c][j][3] *= g4.w;
                p[c][0] = fmaf(S[c][j][0], k4[j].x, p[c][0]); p[c][1] = fmaf(S[c][j][1], k4[j].y, p[c][1]);
                p[c][0] = fmaf(S[c][j][2], k4[j].z, p[c][0]); p[c][1] = fmaf(S[c][j][3], k4[j].w, p[c][1]);
                r[c][0] = fmaf(S[c][j][0], q4.x, r[c][0]); r[c][1] = fmaf(S[c][j][1], q4.y, r[c][1]);
                r[c][0] = fmaf(S[c][j][2], q4.z, r[c][0]); r[c][1] = fmaf(S[c][j][3], q4.w, r[c][1]);
            }
        }
        float u[C];
#pragma unroll
        for (int c = 0; c < C; ++c) {
            float ps = p[c][0] + p[c][1], rs = r[c][0] + r[c][1];
#pragma unroll
            for (int w = LANES / 2; w > 0; w >>= 1) {
                ps += __shfl_xor_sync(0xffffffffu, ps, w);
                rs += __shfl_xor_sync(0xffffffffu, rs, w);
            }
            u[c] = beta * (v[c] - ps);
            o[c] = fmaf(u[c], kq, rs);
        }
#pragma unroll
        for (int j = 0; j < RPL4; ++j)
#pragma unroll
            for (int c = 0; c < C; ++c) {
                S[c][j][0] = fmaf(k4[j].x, u[c], S[c][j][0]); S[c][j][1] = fmaf(k4[j].y, u[c], S[c][j][1]);
                S[c][j][2] = fmaf(k4[j].z, u[c], S[c][j][2]); S[c][j][3] = fmaf(k4[j].w, u[c], S[c][j][3]);
            }
    }
};

// One CTA per (sequence, head, block of C * NT / LANES columns); the C columns of a lane group are GROUPS apart.  TB tokens at a time go
// through shared memory, the next tile is fetched into registers meanwhile.
template <int LANES, int RPL4, int C, int TB, int NT, int UNROLL>
__global__ void __launch_bounds__(NT) delta_scan_kernel(DeltaArgs a) {
    using Col = DeltaColumn<LANES, RPL4>;
    constexpr int D = Col::DMAX, R = TB * D / NT, GROUPS = NT / LANES, COLS = C * GROUPS, RV = (TB * COLS + NT - 1) / NT;
    static_assert(TB * D % NT == 0, "tile shape");
    __shared__ __align__(16) float gs[TB][D], ks[TB][D], qs[TB][D];
    __shared__ float vs[TB][COLS], os[TB][COLS], bs[TB], kqs[TB];
    const int b = blockIdx.x / a.H, h = blockIdx.x % a.H, kvh = h / (a.H / a.G);
    const int l = threadIdx.x % LANES, cl = threadIdx.x / LANES, c0 = blockIdx.y * COLS;
    const int t0 = a.q_start[b], t1 = a.q_start[b + 1], Nk = a.G * a.d, Hd = a.H * a.d, He = a.H * a.e;
    if (t0 >= t1) return;
    float* head = a.state + ((size_t)a.slots[b] * a.H + h) * a.e * a.d;
    float S[C][RPL4][4];
    const bool old = a.seqpos[b] > 0;
#pragma unroll
    for (int c = 0; c < C; ++c) {
        const int col = c0 + c * GROUPS + cl;
        if (old && col < a.e) Col::load(head + (size_t)col * a.d, a.d, l, S[c]);
        else {
#pragma unroll
            for (int j = 0; j < RPL4; ++j) S[c][j][0] = S[c][j][1] = S[c][j][2] = S[c][j][3] = 0.f;
        }
    }
    float pq[R], pk[R], pg[R], pv[RV], pb = 0.f, pkq = 0.f;
    auto fetch = [&](int tb) {
#pragma unroll
        for (int r = 0; r < R; ++r) {
            const int idx = threadIdx.x + r * NT, tt = idx / D, i = idx % D;
            const bool ok = tb + tt < t1 && i < a.d;
            const float* src = a.qk + (size_t)(tb + tt) * 2 * Nk + kvh * a.d + i;
            pq[r] = ok ? src[0] : 0.f;
            pk[r] = ok ? src[Nk] : 0.f;
            pg[r] = ok ? a.g[(size_t)(tb + tt) * Hd + h * a.d + i] : 1.f;  // past the end: nothing forgotten, nothing written
        }
#pragma unroll
        for (int r = 0; r < RV; ++r) {
            const int idx = threadIdx.x + r * NT, tt = idx / COLS, cc = c0 + idx % COLS;
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
            const int idx = threadIdx.x + r * NT, tt = idx / D, i = idx % D;
            gs[tt][i] = pg[r]; ks[tt][i] = pk[r]; qs[tt][i] = pq[r];
        }
#pragma unroll
        for (int r = 0; r < RV; ++r) {
            const int idx = threadIdx.x + r * NT;
            if (idx < TB * COLS) vs[idx / COLS][idx % COLS] = pv[r];
        }
        if (threadIdx.x < TB) { bs[threadIdx.x] = pb; kqs[threadIdx.x] = pkq; }
        __syncthreads();
        if (tb + TB < t1) fetch(tb + TB);
#pragma unroll UNROLL
        for (int tt = 0; tt < TB; ++tt) {  // always the whole tile, so that the next token's operands are read while this one is reduced
            float v[C], o[C];
#pragma unroll
            for (int c = 0; c < C; ++c) v[c] = vs[tt][c * GROUPS + cl];
            Col::template token<C>(gs[tt], ks[tt], qs[tt], kqs[tt], v, bs[tt], l, S, o);
            if (l == 0) {
#pragma unroll
                for (int c = 0; c < C; ++c) os[tt][c * GROUPS + cl] = o[c];
            }
        }
        __syncthreads();
#pragma unroll
        for (int r = 0; r < RV; ++r) {
            const int idx = threadIdx.x + r * NT, tt = idx / COLS, cc = c0 + idx % COLS;
            if (tt < nt && cc < a.e) a.o[(size_t)(tb + tt) * He + h * a.e + cc] = os[tt][idx % COLS];
        }
    }
#pragma unroll
    for (int c = 0; c < C; ++c) {
        const int col = c0 + c * GROUPS + cl;
        if (col < a.e) Col::store(head + (size_t)col * a.d, a.d, l, S[c]);
    }
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

__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}

// One CTA per (sequence, head), one token: convolutions and unit norms, decays (second half of their low-rank projection included), beta, the
// state update and read-out, the head's norm, and the output gate (second half of its projection included).  Every load that depends on
// nothing (state of the first columns, slices of the second projections, carried inputs) is issued first.  Shared memory:
// qs ks gs [DMAX] | v gate o [e] | decay latent [ra] | gate latent [rg] | with a.stage: the head's rows of w_a2 [d, ra] and w_g2 [e, rg]
template <typename T, int LANES, int RPL4, int MIN_CTAS>
__global__ void __launch_bounds__(DT_THREADS, MIN_CTAS) delta_step_kernel(DeltaArgs a) {
    using Col = DeltaColumn<LANES, RPL4>;
    constexpr int D = Col::DMAX, GROUPS = DT_THREADS / LANES;
    extern __shared__ __align__(16) float dsm[];
    float *qs = dsm, *ks = qs + D, *gs = ks + D, *vs = gs + D, *gate = vs + a.e, *os = gate + a.e, *la = os + a.e, *lg = la + a.ra;
    __shared__ float red[32], sc[3];
    const int b = blockIdx.x / a.H, h = blockIdx.x % a.H, rep = a.H / a.G, kvh = h / rep, tid = threadIdx.x;
    const int Nk = a.G * a.d, channels = 2 * Nk + a.H * a.e, pos = a.positions[b], slot = a.slots[b];
    const int l = tid % LANES, cl = tid / LANES;
    const T* wa = static_cast<const T*>(a.w_a2) + (size_t)h * a.d * a.ra;
    const T* wg = static_cast<const T*>(a.w_g2) + (size_t)h * a.e * a.rg;
    if (a.stage) {
        constexpr int V = 16 / sizeof(T);
        T* stage = reinterpret_cast<T*>((reinterpret_cast<uintptr_t>(lg + a.rg) + 15) & ~(uintptr_t)15);
        const int na = a.d * a.ra, ng = a.e * a.rg;
        for (int i = tid * V; i < na; i += DT_THREADS * V) cp_async16(stage + i, wa + i);
        for (int i = tid * V; i < ng; i += DT_THREADS * V) cp_async16(stage + na + i, wg + i);
        wa = stage;
        wg = stage + na;
    }
    asm volatile("cp.async.commit_group;\n");
    float* head = a.state + ((size_t)slot * a.H + h) * a.e * a.d;
    const bool old = a.seqpos[b] > 0;
    float S[DT_PASS][RPL4][4];
    auto load_state = [&](int c0) {
#pragma unroll
        for (int p = 0; p < DT_PASS; ++p) {
            const int c = c0 + p * GROUPS + cl;
            if (old && c < a.e) Col::load(head + (size_t)c * a.d, a.d, l, S[p]);
            else {
#pragma unroll
                for (int j = 0; j < RPL4; ++j) S[p][j][0] = S[p][j][1] = S[p][j][2] = S[p][j][3] = 0.f;
            }
        }
    };
    load_state(0);
    const T* row = static_cast<const T*>(a.y) + (size_t)b * a.y_pitch;
    for (int i = tid; i < a.ra; i += DT_THREADS) la[i] = to_f(row[channels + a.H + i]);
    for (int i = tid; i < a.rg; i += DT_THREADS) lg[i] = to_f(row[channels + a.H + a.ra + i]);
    const float beta = sigmoid_exact(to_f(row[channels + h]));
    float* cs = a.cstate + (size_t)slot * a.taps * channels;
    for (int i = tid; i < 2 * D + a.e; i += DT_THREADS) {
        const int which = i < D ? 0 : i < 2 * D ? 1 : 2, c = i - which * D;
        if (which < 2 && c >= a.d) { (which ? ks : qs)[c] = 0.f; continue; }
        const int ch = which == 0 ? kvh * a.d + c : which == 1 ? Nk + kvh * a.d + c : 2 * Nk + h * a.e + c;
        const T* w = static_cast<const T*>(a.conv) + (size_t)ch * a.taps;
        const float x = to_f(row[ch]);
        float acc = to_f(w[a.taps - 1]) * x;
        int back = 1;
        for (; back + 2 < a.taps; back += 3) {  // three carried inputs in flight
            float xv[3];
#pragma unroll
            for (int u = 0; u < 3; ++u) xv[u] = back + u <= pos ? cs[(size_t)((pos - back - u) % a.taps) * channels + ch] : 0.f;
#pragma unroll
            for (int u = 0; u < 3; ++u) acc = fmaf(to_f(w[a.taps - 1 - back - u]), xv[u], acc);
        }
        for (; back < a.taps; ++back)
            if (back <= pos) acc = fmaf(to_f(w[a.taps - 1 - back]), cs[(size_t)((pos - back) % a.taps) * channels + ch], acc);
        (which == 0 ? qs : which == 1 ? ks : vs)[c] = silu_exact(acc);
        if (a.taps > 1 && (which == 2 || h % rep == 0)) cs[(size_t)(pos % a.taps) * channels + ch] = x;
    }
    asm volatile("cp.async.wait_group 0;\n");
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
            const float s = dot8<T>(is_d ? wa + (size_t)r * a.ra : wg + (size_t)(live ? r - a.d : 0) * a.rg, is_d ? la : lg, is_d ? a.ra : a.rg, l8);
            if (live && l8 == 0) {
                if (is_d) gs[r] = delta_decay(s + to_f(static_cast<const T*>(a.dt_bias)[h * a.d + r]), alog);
                else gate[r - a.d] = sigmoid_exact(rnd<T>(s));
            }
        }
        for (int i = a.d + tid; i < D; i += DT_THREADS) gs[i] = 0.f;
    }
    __syncthreads();
    const float iq = sc[0], ik = sc[1], kq = sc[2] * iq * ik;
    for (int i = tid; i < D; i += DT_THREADS) {
        ks[i] *= ik;
        qs[i] *= iq;
    }
    __syncthreads();
    for (int c0 = 0; c0 < a.e; c0 += DT_PASS * GROUPS) {
        if (c0 > 0) load_state(c0);
        float v[DT_PASS], o[DT_PASS];
#pragma unroll
        for (int p = 0; p < DT_PASS; ++p) {
            const int c = c0 + p * GROUPS + cl;
            v[p] = c < a.e ? vs[c] : 0.f;
        }
        Col::template token<DT_PASS>(gs, ks, qs, kq, v, beta, l, S, o);
#pragma unroll
        for (int p = 0; p < DT_PASS; ++p) {
            const int c = c0 + p * GROUPS + cl;
            if (c < a.e) {
                if (l == 0) os[c] = o[p];
                Col::store(head + (size_t)c * a.d, a.d, l, S[p]);
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
