// Decode attention on tensor cores (bf16 storage): one token per sequence, every key and value row read once for all query heads of its group.
//
// grid (sequence * key/value head, splits), four warps.  The (up to 16) query heads of the group are the M side of m16n8k16 tiles; every warp walks
// its own 16-key pieces of the ring (pieces are dealt out over warps and splits) with its own running (max, sum) and value accumulators, its
// pieces arriving by cp.async in a private ring of DA_STAGES buffers -- warps never wait for one another before the end, when they are merged
// through shared memory.  The splits' partial results have the layout of attn_bias_kernel's and go through the same merge kernels (sinks,
// differences of two maps, gates).  With MAPS 2 both maps of a head are computed here: their keys are one row, their values are shared.
#pragma once
#include "hybrid_attn_flash.cuh"

namespace mbh {

constexpr int DA_WARPS = 4, DA_KEYS = 16, DA_STAGES = 3, DA_MAX_GROUP = 16;

template <int D, int E, int MAPS> constexpr size_t attn_decode_smem() {
    constexpr size_t stages = sizeof(bf16) * (size_t)DA_WARPS * DA_STAGES * DA_KEYS * (MAPS * D + 8 + E + 8);
    constexpr size_t merge = sizeof(float) * (size_t)DA_WARPS * MAPS * 16 * (E + 2);
    return stages > merge ? stages : merge;
}

template <int D, int E, int MAPS>
__global__ void __launch_bounds__(DA_WARPS * 32) attn_decode_mma_kernel(AttnArgs a) {
    constexpr int KP = MAPS * D + 8, VP = E + 8, STAGE = DA_KEYS * (KP + VP);
    constexpr float LOG2E = 1.4426950408889634f, LN2 = 0.6931471805599453f;
    extern __shared__ __align__(16) unsigned char da_smem[];
    const int b = blockIdx.x / a.G, g = blockIdx.x % a.G, R = a.H / a.G, split = blockIdx.y;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
    bf16* const mine = reinterpret_cast<bf16*>(da_smem) + warp * DA_STAGES * STAGE;
    const int pos = a.positions[b], lo = first_key(a, pos);
    const size_t base = (size_t)a.slots[b] * a.W, kstride = (size_t)a.G * MAPS * D, vstride = (size_t)a.G * E;
    const bf16* K = static_cast<const bf16*>(a.cache_k) + base * kstride + (size_t)g * MAPS * D;
    const bf16* V = static_cast<const bf16*>(a.cache_v) + base * vstride + (size_t)g * E;
    const bf16* Q = static_cast<const bf16*>(a.q) + ((size_t)b * a.H + g * R) * MAPS * D;

    const int step = a.splits * DA_WARPS * DA_KEYS;
    auto load = [&](int c0, int stage) {  // keys c0 .. c0 + 15 (those up to pos)
        bf16* ks = mine + stage * STAGE;
        bf16* vs = ks + DA_KEYS * KP;
        if (c0 <= pos) {
            const int s0 = c0 % a.W;
            constexpr int CK = MAPS * D / 8, CV = E / 8;
#pragma unroll
            for (int c = lane; c < DA_KEYS * CK; c += 32) {
                const int r = c / CK, kc = (c % CK) * 8, s = s0 + r;
                const bool ok = c0 + r <= pos;
                cp_async16(ks + r * KP + kc, ok ? K + (size_t)(s < a.W ? s : s % a.W) * kstride + kc : K, ok);
            }
#pragma unroll
            for (int c = lane; c < DA_KEYS * CV; c += 32) {
                const int r = c / CV, ec = (c % CV) * 8, s = s0 + r;
                const bool ok = c0 + r <= pos;
                cp_async16(vs + r * VP + ec, ok ? V + (size_t)(s < a.W ? s : s % a.W) * vstride + ec : V, ok);
            }
        }
        cp_async_commit();
    };
    const int first = lo + (split * DA_WARPS + warp) * DA_KEYS;
#pragma unroll
    for (int i = 0; i < DA_STAGES - 1; ++i) load(first + i * step, i);

    uint32_t qf[MAPS][D / 16][4];
#pragma unroll
    for (int m = 0; m < MAPS; ++m)
#pragma unroll
        for (int kk = 0; kk < D / 16; ++kk)
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const int row = gid + (u & 1) * 8, col = kk * 16 + tig * 2 + (u >> 1) * 8;
                qf[m][kk][u] = row < R ? *reinterpret_cast<const uint32_t*>(Q + ((size_t)row * MAPS + m) * D + col) : 0u;
            }
    float o[MAPS][E / 8][4], mx[MAPS][2], l[MAPS][2];  // maxima in units of log2
#pragma unroll
    for (int m = 0; m < MAPS; ++m) {
        mx[m][0] = mx[m][1] = -INFINITY; l[m][0] = l[m][1] = 0.f;
#pragma unroll
        for (int ne = 0; ne < E / 8; ++ne) o[m][ne][0] = o[m][ne][1] = o[m][ne][2] = o[m][ne][3] = 0.f;
    }
    const bool capped = a.softcap > 0.f;
    const float unit = (capped ? 1.f : a.scale) * LOG2E, capf = capped ? 2.f * a.scale / a.softcap : 0.f;

    int stage = 0;
    for (int c0 = first; c0 <= pos; c0 += step) {
        load(c0 + (DA_STAGES - 1) * step, (stage + DA_STAGES - 1) % DA_STAGES);
        cp_async_wait<DA_STAGES - 1>();
        __syncwarp();
        const bf16* ks = mine + stage * STAGE;
        const bf16* vs = ks + DA_KEYS * KP;
        uint32_t pa[MAPS][4];
#pragma unroll
        for (int m = 0; m < MAPS; ++m) {
            float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
            const bf16* kp = ks + ((lane >> 4) * 8 + (lane & 7)) * KP + m * D + ((lane >> 3) & 1) * 8;
#pragma unroll
            for (int kk = 0; kk < D / 16; ++kk) {
                uint32_t kf[4];
                ldmatrix4(kf, kp + kk * 16);
                mma_bf16(s[0], qf[m][kk], kf[0], kf[1]);
                mma_bf16(s[1], qf[m][kk], kf[2], kf[3]);
            }
            float t0 = -INFINITY, t1 = -INFINITY;
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int c = 0; c < 2; ++c) {
                    const bool ok = c0 + nt * 8 + tig * 2 + c <= pos;
                    float x0 = s[nt][c], x1 = s[nt][2 + c];
                    if (capped) { x0 = softcap_fast(x0, a.softcap, capf); x1 = softcap_fast(x1, a.softcap, capf); }
                    s[nt][c] = ok ? x0 * unit : -INFINITY; s[nt][2 + c] = ok ? x1 * unit : -INFINITY;
                    t0 = fmaxf(t0, s[nt][c]); t1 = fmaxf(t1, s[nt][2 + c]);
                }
            // key c0 is visible, so the new maxima are finite
            t0 = fmaxf(mx[m][0], quad_max(t0)); t1 = fmaxf(mx[m][1], quad_max(t1));
            const float f0 = exp2_fast(mx[m][0] - t0), f1 = exp2_fast(mx[m][1] - t1);
            mx[m][0] = t0; mx[m][1] = t1;
            float q0 = 0.f, q1 = 0.f;
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int c = 0; c < 2; ++c) {
                    s[nt][c] = exp2_fast(s[nt][c] - t0); s[nt][2 + c] = exp2_fast(s[nt][2 + c] - t1);
                    q0 += s[nt][c]; q1 += s[nt][2 + c];
                }
            l[m][0] = l[m][0] * f0 + q0; l[m][1] = l[m][1] * f1 + q1;
#pragma unroll
            for (int ne = 0; ne < E / 8; ++ne) { o[m][ne][0] *= f0; o[m][ne][1] *= f0; o[m][ne][2] *= f1; o[m][ne][3] *= f1; }
            pa[m][0] = pack_bf16(s[0][0], s[0][1]); pa[m][1] = pack_bf16(s[0][2], s[0][3]);
            pa[m][2] = pack_bf16(s[1][0], s[1][1]); pa[m][3] = pack_bf16(s[1][2], s[1][3]);
        }
        const bf16* vp = vs + (((lane >> 3) & 1) * 8 + (lane & 7)) * VP + (lane >> 4) * 8;
#pragma unroll
        for (int np = 0; np < E / 16; ++np) {
            uint32_t vf[4];
            ldmatrix4_trans(vf, vp + np * 16);
#pragma unroll
            for (int m = 0; m < MAPS; ++m) {
                mma_bf16(o[m][2 * np], pa[m], vf[0], vf[1]);
                mma_bf16(o[m][2 * np + 1], pa[m], vf[2], vf[3]);
            }
        }
        __syncwarp();  // the buffer is used up
        stage = (stage + 1) % DA_STAGES;
    }
    cp_async_wait<0>();
    __syncthreads();
    // the warps' results: [warp][map][row] of (max, sum, E values)
    float* mrg = reinterpret_cast<float*>(da_smem);
#pragma unroll
    for (int m = 0; m < MAPS; ++m) {
        float* p0 = mrg + ((size_t)(warp * MAPS + m) * 16 + gid) * (E + 2);
        float* p1 = p0 + 8 * (E + 2);
        const float s0 = quad_sum(l[m][0]), s1 = quad_sum(l[m][1]);
        if (tig == 0) { p0[0] = mx[m][0]; p0[1] = s0; p1[0] = mx[m][1]; p1[1] = s1; }
#pragma unroll
        for (int ne = 0; ne < E / 8; ++ne) {
            const int col = 2 + ne * 8 + tig * 2;
            *reinterpret_cast<float2*>(p0 + col) = make_float2(o[m][ne][0], o[m][ne][1]);
            *reinterpret_cast<float2*>(p1 + col) = make_float2(o[m][ne][2], o[m][ne][3]);
        }
    }
    __syncthreads();
    for (int rm = warp; rm < R * MAPS; rm += DA_WARPS) {  // a warp per (query head, map)
        const int row = rm / MAPS, m = rm % MAPS;
        const float* p = mrg + ((size_t)m * 16 + row) * (E + 2);
        constexpr size_t WS = (size_t)MAPS * 16 * (E + 2);
        float M = -INFINITY, L = 0.f, f[DA_WARPS];
#pragma unroll
        for (int w = 0; w < DA_WARPS; ++w) M = fmaxf(M, p[w * WS]);
#pragma unroll
        for (int w = 0; w < DA_WARPS; ++w) {
            f[w] = p[w * WS] == -INFINITY ? 0.f : exp2_fast(p[w * WS] - M);
            L += f[w] * p[w * WS + 1];
        }
        float* out = a.scratch + ((((size_t)b * a.H + g * R + row) * MAPS + m) * a.splits + split) * (2 + E);
        if (lane == 0) { out[0] = M * LN2; out[1] = L; }
        for (int c = lane; c < E; c += 32) {
            float v = 0.f;
#pragma unroll
            for (int w = 0; w < DA_WARPS; ++w) v = fmaf(f[w], p[w * WS + 2 + c], v);
            out[2 + c] = v;
        }
    }
}

template <int D, int E, int MAPS> inline cudaError_t run_attn_decode(const AttnArgs& a, cudaStream_t st) {
    constexpr size_t smem = attn_decode_smem<D, E, MAPS>();
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(attn_decode_mma_kernel<D, E, MAPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e) return e;
    }
    attn_decode_mma_kernel<D, E, MAPS><<<dim3((unsigned)(a.B * a.G), (unsigned)a.splits), DA_WARPS * 32, smem, st>>>(a);
    return cudaGetLastError();
}

// true when a (D, E, maps) instantiation exists; launches it (partial results only)
inline bool launch_attn_decode(const AttnArgs& a, cudaStream_t st, cudaError_t& err) {
    if (a.H / a.G > DA_MAX_GROUP) return false;
#define MBH_DA(DD, EE, MM) if (a.d == DD && a.e == EE && a.maps == MM) { err = run_attn_decode<DD, EE, MM>(a, st); return true; }
    MBH_DA(32, 32, 1) MBH_DA(64, 32, 1) MBH_DA(64, 64, 1) MBH_DA(64, 128, 1) MBH_DA(128, 64, 1) MBH_DA(128, 128, 1) MBH_DA(96, 64, 1) MBH_DA(96, 96, 1)
    MBH_DA(32, 32, 2) MBH_DA(32, 64, 2) MBH_DA(48, 96, 2) MBH_DA(64, 64, 2) MBH_DA(64, 128, 2) MBH_DA(96, 96, 2) MBH_DA(128, 128, 2)
#undef MBH_DA
    return false;
}

}  // namespace mbh
