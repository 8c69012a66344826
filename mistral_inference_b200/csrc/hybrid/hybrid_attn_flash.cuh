// Prompt attention on tensor cores (bf16 storage): flash-style, one CTA per (64-query tile, head).
//
// Four warps, 16 queries each.  Tiles of 64 keys and values come from the layer's ring or from the call's own rows into shared memory by
// cp.async, two stages, the next tile in flight while this one is used; rows are padded by 16 bytes, so that ldmatrix (transposing for the
// values) meets no bank conflict.  S = Q K^T with mma.sync.m16n8k16 (Q fragments stay in registers); scores times the scale, with an
// optional additive bias[min(distance, n_tab - 1), h]; masks are applied on the tiles that a row's first key or the diagonal cuts; running
// (max, sum) per query row in fp32, exponentials base 2; P is rounded to bf16 and multiplies V with fp32 accumulators.  Query tiles never straddle
// two sequences; positions inside a tile are consecutive.  The longest tiles start first.
// AttnArgs::softcap and AttnArgs::sink as in attn_bias_kernel (the cap's tanh through one fast exponential).
// With AttnArgs::sigmoid the weights are sigmoid(score) (fp32, then bf16 for P V) and nothing is normalised.
// MAPS 2 (differential attention): eight warps, four per map; every map has its own keys, the values are staged once for both.  The second
// map's normalised result goes through shared memory to the first map's warps, which subtract, norm and write.
// Chunks and output gates as in attn_bias_kernel.
#pragma once
#include "hybrid_mixers.cuh"

namespace mbh {

__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&v);
}
__device__ __forceinline__ float quad_max(float v) {
    v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 1));
    return fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 2));
}
__device__ __forceinline__ float quad_sum(float v) {
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    return v + __shfl_xor_sync(0xffffffffu, v, 2);
}

constexpr int FA_BQ = 64, FA_BK = 64;

__device__ __forceinline__ void ldmatrix4(uint32_t* r, const bf16* p) {
    const uint32_t addr = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix4_trans(uint32_t* r, const bf16* p) {
    const uint32_t addr = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
// 16 bytes to shared memory, zeros when !ok (src is then not read)
__device__ __forceinline__ void cp_async16(bf16* dst, const bf16* src, bool ok) {
    const uint32_t addr = (uint32_t)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(addr), "l"(src), "r"(ok ? 16 : 0));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N)); }
__device__ __forceinline__ float exp2_fast(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}

// dynamic shared memory: two stages of keys [MAPS][64][D + 8] and values [64][E + 8] (bf16); afterwards the second map's result [64][E + 4] (fp32)
template <int D, int E, int MAPS> constexpr size_t attn_flash_smem() {
    constexpr size_t tiles = 2 * sizeof(bf16) * (size_t)(MAPS * FA_BK * (D + 8) + FA_BK * (E + 8)), other = MAPS > 1 ? sizeof(float) * (size_t)FA_BQ * (E + 4) : 0;
    return tiles > other ? tiles : other;
}

template <int D, int E, int MAPS>
__global__ void __launch_bounds__(128 * MAPS) attn_bias_flash_kernel(AttnArgs a) {
    constexpr int KP = D + 8, VP = E + 8, NT = 128 * MAPS, STAGE = MAPS * FA_BK * KP + FA_BK * VP;
    constexpr float LOG2E = 1.4426950408889634f, LN2 = 0.6931471805599453f;
    extern __shared__ __align__(16) unsigned char fa_smem[];
    bf16* const stages = reinterpret_cast<bf16*>(fa_smem);  // per stage: map m's key r in row m * FA_BK + r (pitch KP), then the values (pitch VP)
    const int h = blockIdx.y, g = h / (a.H / a.G);
    int tile = gridDim.x - 1 - blockIdx.x, b = 0, t0 = 0;
    for (; b < a.B; ++b) {
        const int len = a.q_start[b + 1] - a.q_start[b], nt = (len + FA_BQ - 1) / FA_BQ;
        if (tile < nt) { t0 = a.q_start[b] + tile * FA_BQ; break; }
        tile -= nt;
    }
    if (b == a.B) return;
    const int t_end = a.q_start[b + 1];
    const int warp = (threadIdx.x >> 5) & 3, map = threadIdx.x >> 7, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
    const int r0 = t0 + warp * 16 + gid, r1 = r0 + 8;
    const bool v0 = r0 < t_end, v1 = r1 < t_end;
    const int pos_first = a.positions[t0];
    const int p0 = v0 ? pos_first + (r0 - t0) : -1, p1 = v1 ? pos_first + (r1 - t0) : -1;
    const int pos_last = pos_first + (min(t0 + FA_BQ, t_end) - 1 - t0);
    const int pos_warp = pos_first + warp * 16;                                        // of the warp's first row
    const int pos_warp_last = pos_first + (min(t0 + warp * 16 + 16, t_end) - 1 - t0);  // below pos_warp when the warp has no row

    const bf16* Q = static_cast<const bf16*>(a.q);
    uint32_t qf[D / 16][4];
#pragma unroll
    for (int ks = 0; ks < D / 16; ++ks) {
        const int col = ks * 16 + tig * 2;
        const bf16* q0 = Q + (((size_t)r0 * a.H + h) * MAPS + map) * D + col;
        const bf16* q1 = Q + (((size_t)r1 * a.H + h) * MAPS + map) * D + col;
        qf[ks][0] = v0 ? *reinterpret_cast<const uint32_t*>(q0) : 0u;
        qf[ks][1] = v1 ? *reinterpret_cast<const uint32_t*>(q1) : 0u;
        qf[ks][2] = v0 ? *reinterpret_cast<const uint32_t*>(q0 + 8) : 0u;
        qf[ks][3] = v1 ? *reinterpret_cast<const uint32_t*>(q1 + 8) : 0u;
    }
    float o[E / 8][4];
#pragma unroll
    for (int ne = 0; ne < E / 8; ++ne) o[ne][0] = o[ne][1] = o[ne][2] = o[ne][3] = 0.f;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;  // maxima in units of log2
    const size_t base = (size_t)a.slots[b] * a.W;
    const size_t kstride = (size_t)a.G * MAPS * D, vstride = (size_t)a.G * E;
    const int own_from = a.own_k ? a.seqpos[b] : 0x7fffffff;
    const size_t own_row = a.own_k ? (size_t)a.q_start[b] : 0;
    const KeySource<bf16> Ksrc{static_cast<const bf16*>(a.cache_k) + base * kstride + (size_t)g * MAPS * D,
                               static_cast<const bf16*>(a.own_k) + own_row * kstride + (size_t)g * MAPS * D, kstride, kstride, a.W, own_from};
    const KeySource<bf16> Vsrc{static_cast<const bf16*>(a.cache_v) + base * vstride + (size_t)g * E,
                               static_cast<const bf16*>(a.own_v) + own_row * vstride + (size_t)g * E, vstride, vstride, a.W, own_from};
    // window or chunks: the first key any row of this tile sees, key tiles below it are skipped; then those of this warp and of its two rows
    const int j_lo = first_key(a, pos_first), lo_warp = first_key(a, pos_warp), lo_warp_last = first_key(a, pos_warp_last), lo0 = first_key(a, p0), lo1 = first_key(a, p1);
    const float* bias = a.bias_tab ? a.bias_tab + h : nullptr;  // null: no bias
    const int last_tab = a.n_tab - 1;
    const bool capped = a.softcap > 0.f, plain = !bias && !a.sigmoid;
    const float scale = capped ? 1.f : a.scale;  // a capped score has its scale inside the cap
    const float unit = scale * (plain ? LOG2E : 1.f);

    auto load = [&](int j0, int stage) {
        bf16* ks = stages + stage * STAGE;
        bf16* vs = ks + MAPS * FA_BK * KP;
        constexpr int CK = MAPS * D / 8, CV = E / 8;  // a key row holds the keys of all maps
#pragma unroll 4
        for (int c = threadIdx.x; c < FA_BK * CK; c += NT) {
            const int r = c / CK, kc = (c % CK) * 8, j = j0 + r;
            const bool ok = j <= pos_last && j >= j_lo;
            cp_async16(ks + ((MAPS > 1 ? kc / D : 0) * FA_BK + r) * KP + (MAPS > 1 ? kc % D : kc), ok ? Ksrc.row(j) + kc : Q, ok);
        }
#pragma unroll 4
        for (int c = threadIdx.x; c < FA_BK * CV; c += NT) {
            const int r = c / CV, ec = (c % CV) * 8, j = j0 + r;
            const bool ok = j <= pos_last && j >= j_lo;
            cp_async16(vs + r * VP + ec, ok ? Vsrc.row(j) + ec : Q, ok);
        }
        cp_async_commit();
    };

    int stage = 0;
    const int j_start = (j_lo / FA_BK) * FA_BK;
    load(j_start, 0);
    for (int j0 = j_start; j0 <= pos_last; j0 += FA_BK, stage ^= 1) {
        if (j0 + FA_BK <= pos_last) { load(j0 + FA_BK, stage ^ 1); cp_async_wait<1>(); }
        else cp_async_wait<0>();
        __syncthreads();
        // skipped: every key of this tile is in the future of this warp's rows, or before what they see
        if (j0 <= pos_warp_last && j0 + FA_BK > lo_warp) {
            const bf16* ks = stages + stage * STAGE + map * FA_BK * KP;
            const bf16* vs = stages + stage * STAGE + MAPS * FA_BK * KP;
            float s[8][4];
#pragma unroll
            for (int nt = 0; nt < 8; ++nt) s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.f;
            const bf16* kp = ks + ((lane >> 4) * 8 + (lane & 7)) * KP + ((lane >> 3) & 1) * 8;
#pragma unroll
            for (int kk = 0; kk < D / 16; ++kk)
#pragma unroll
                for (int np = 0; np < 4; ++np) {
                    uint32_t kf[4];
                    ldmatrix4(kf, kp + np * 16 * KP + kk * 16);
                    mma_bf16(s[2 * np], qf[kk], kf[0], kf[1]);
                    mma_bf16(s[2 * np + 1], qf[kk], kf[2], kf[3]);
                }
            if (capped) {
                const float f = 2.f * a.scale / a.softcap;
#pragma unroll
                for (int nt = 0; nt < 8; ++nt)
#pragma unroll
                    for (int c = 0; c < 4; ++c) s[nt][c] = softcap_fast(s[nt][c], a.softcap, f);
            }
            float mx0 = -INFINITY, mx1 = -INFINITY;
            if (plain && j0 + FA_BK - 1 <= pos_warp && j0 >= lo_warp_last) {  // every row of the warp sees every key of the tile
#pragma unroll
                for (int nt = 0; nt < 8; ++nt)
#pragma unroll
                    for (int c = 0; c < 2; ++c) {
                        s[nt][c] *= unit; s[nt][2 + c] *= unit;
                        mx0 = fmaxf(mx0, s[nt][c]); mx1 = fmaxf(mx1, s[nt][2 + c]);
                    }
            } else {
#pragma unroll
                for (int nt = 0; nt < 8; ++nt)
#pragma unroll
                    for (int c = 0; c < 2; ++c) {
                        const int j = j0 + nt * 8 + tig * 2 + c;
                        float x0 = s[nt][c] * unit, x1 = s[nt][2 + c] * unit;
                        if (bias) { x0 += bias[(size_t)min(max(p0 - j, 0), last_tab) * a.H]; x1 += bias[(size_t)min(max(p1 - j, 0), last_tab) * a.H]; }
                        if (!plain && !a.sigmoid) { x0 *= LOG2E; x1 *= LOG2E; }
                        x0 = (j <= p0 && j >= lo0) ? x0 : -INFINITY;
                        x1 = (j <= p1 && j >= lo1) ? x1 : -INFINITY;
                        s[nt][c] = x0; s[nt][2 + c] = x1;
                        mx0 = fmaxf(mx0, x0); mx1 = fmaxf(mx1, x1);
                    }
            }
            float ps0 = 0.f, ps1 = 0.f;
            if (a.sigmoid) {  // weights sigmoid(score), 0 where masked; nothing to rescale
#pragma unroll
                for (int nt = 0; nt < 8; ++nt)
#pragma unroll
                    for (int c = 0; c < 4; ++c) s[nt][c] = s[nt][c] == -INFINITY ? 0.f : __fdividef(1.f, 1.f + __expf(-s[nt][c]));  // rounded to bf16 just below
            } else {
                const float mn0 = fmaxf(m0, quad_max(mx0)), mn1 = fmaxf(m1, quad_max(mx1));
                const float z0 = mn0 == -INFINITY ? 0.f : mn0, z1 = mn1 == -INFINITY ? 0.f : mn1;  // a row that has seen no key yet: all weights 2^-inf = 0
                const float c0 = exp2_fast(m0 - z0), c1 = exp2_fast(m1 - z1);
#pragma unroll
                for (int nt = 0; nt < 8; ++nt)
#pragma unroll
                    for (int c = 0; c < 2; ++c) {
                        s[nt][c] = exp2_fast(s[nt][c] - z0); s[nt][2 + c] = exp2_fast(s[nt][2 + c] - z1);
                        ps0 += s[nt][c]; ps1 += s[nt][2 + c];
                    }
                l0 = l0 * c0 + ps0; l1 = l1 * c1 + ps1;  // per-thread partial sums; the quad is reduced at the end (same factors in a quad)
                m0 = mn0; m1 = mn1;
#pragma unroll
                for (int ne = 0; ne < E / 8; ++ne) { o[ne][0] *= c0; o[ne][1] *= c0; o[ne][2] *= c1; o[ne][3] *= c1; }
            }
            const bf16* vp = vs + (((lane >> 3) & 1) * 8 + (lane & 7)) * VP + (lane >> 4) * 8;
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) {
                const uint32_t pa[4] = {pack_bf16(s[2 * kk][0], s[2 * kk][1]), pack_bf16(s[2 * kk][2], s[2 * kk][3]),
                                        pack_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1]), pack_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3])};
#pragma unroll
                for (int np = 0; np < E / 16; ++np) {
                    uint32_t vf[4];
                    ldmatrix4_trans(vf, vp + kk * 16 * VP + np * 16);
                    mma_bf16(o[2 * np], pa, vf[0], vf[1]);
                    mma_bf16(o[2 * np + 1], pa, vf[2], vf[3]);
                }
            }
        }
        __syncthreads();  // the tile is used up: its stage takes the one after the next
    }
    l0 = quad_sum(l0); l1 = quad_sum(l1);
    if (a.sigmoid) l0 = l1 = 1.f;
    if (a.sink) { l0 = sink_denominator(m0 * LN2, l0, a.sink[h]); l1 = sink_denominator(m1 * LN2, l1, a.sink[h]); }
    float f0 = 1.f / l0, f1 = 1.f / l1;  // rows past the end hold nothing useful and are not written
    if constexpr (MAPS > 1) {
        float (*X)[E + 4] = reinterpret_cast<float (*)[E + 4]>(fa_smem);
        const int x0 = warp * 16 + gid, x1 = x0 + 8;
        if (map == 1) {  // the last barrier of the loop has freed the tiles' memory
            const float lam = *a.lambda;
#pragma unroll
            for (int ne = 0; ne < E / 8; ++ne) {
                const int col = ne * 8 + tig * 2;
                *reinterpret_cast<float2*>(&X[x0][col]) = make_float2(lam * (o[ne][0] * f0), lam * (o[ne][1] * f0));
                *reinterpret_cast<float2*>(&X[x1][col]) = make_float2(lam * (o[ne][2] * f1), lam * (o[ne][3] * f1));
            }
        }
        __syncthreads();
        if (map == 1) return;
        float s0 = 0.f, s1 = 0.f;
#pragma unroll
        for (int ne = 0; ne < E / 8; ++ne) {
            const int col = ne * 8 + tig * 2;
            const float2 y0 = *reinterpret_cast<const float2*>(&X[x0][col]), y1 = *reinterpret_cast<const float2*>(&X[x1][col]);
            o[ne][0] = o[ne][0] * f0 - y0.x; o[ne][1] = o[ne][1] * f0 - y0.y;
            o[ne][2] = o[ne][2] * f1 - y1.x; o[ne][3] = o[ne][3] * f1 - y1.y;
            s0 = fmaf(o[ne][0], o[ne][0], fmaf(o[ne][1], o[ne][1], s0));
            s1 = fmaf(o[ne][2], o[ne][2], fmaf(o[ne][3], o[ne][3], s1));
        }
        f0 = a.out_scale / sqrtf(quad_sum(s0) / (float)E + a.norm_eps);
        f1 = a.out_scale / sqrtf(quad_sum(s1) / (float)E + a.norm_eps);
    }
    bf16* out = static_cast<bf16*>(a.out);
    const bf16* gate = static_cast<const bf16*>(a.gate);
    if (gate && !a.gate_entry) {
        if (v0) f0 *= sigmoid_exact(to_f(gate[(size_t)r0 * a.gate_pitch + h]));
        if (v1) f1 *= sigmoid_exact(to_f(gate[(size_t)r1 * a.gate_pitch + h]));
    }
    const bool entry = gate && a.gate_entry;
    auto emit = [&](int r, int col, float x, float y) {
        if (entry) {  // gate_pitch is even with entry gates of even heads (checked by the host)
            const float2 g2 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gate + (size_t)r * a.gate_pitch + h * E + col));
            x *= sigmoid_exact(g2.x); y *= sigmoid_exact(g2.y);
        }
        *reinterpret_cast<__nv_bfloat162*>(out + ((size_t)r * a.H + h) * E + col) = __floats2bfloat162_rn(x, y);
    };
#pragma unroll
    for (int ne = 0; ne < E / 8; ++ne) {
        const int col = ne * 8 + tig * 2;
        if (v0) emit(r0, col, o[ne][0] * f0, o[ne][1] * f0);
        if (v1) emit(r1, col, o[ne][2] * f1, o[ne][3] * f1);
    }
}

template <int D, int E, int MAPS> inline cudaError_t run_attn_flash(const AttnArgs& a, int n_tiles, cudaStream_t st) {
    constexpr size_t smem = attn_flash_smem<D, E, MAPS>();
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(attn_bias_flash_kernel<D, E, MAPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e) return e;
    }
    attn_bias_flash_kernel<D, E, MAPS><<<dim3((unsigned)n_tiles, (unsigned)a.H), 128 * MAPS, smem, st>>>(a);
    return cudaGetLastError();
}

// true when a (D, E) instantiation exists (and the gate's pairs are aligned); launches it
inline bool launch_attn_flash(const AttnArgs& a, int n_tiles, cudaStream_t st, cudaError_t& err) {
    if (a.gate && a.gate_entry && (a.gate_pitch % 2 || reinterpret_cast<uintptr_t>(a.gate) % 4)) return false;
#define MBH_FA2(DD, EE) if (a.maps == 2 && a.d == DD && a.e == EE) { err = run_attn_flash<DD, EE, 2>(a, n_tiles, st); return true; }
    MBH_FA2(32, 32) MBH_FA2(32, 64) MBH_FA2(48, 96) MBH_FA2(64, 64) MBH_FA2(64, 128) MBH_FA2(96, 96) MBH_FA2(128, 128)
#undef MBH_FA2
    if (a.maps != 1) return false;
#define MBH_FA(DD, EE) if (a.d == DD && a.e == EE) { err = run_attn_flash<DD, EE, 1>(a, n_tiles, st); return true; }
    MBH_FA(32, 32) MBH_FA(64, 32) MBH_FA(64, 64) MBH_FA(128, 64) MBH_FA(64, 128) MBH_FA(128, 128) MBH_FA(96, 64) MBH_FA(96, 96) MBH_FA(48, 32) MBH_FA(192, 128)
#undef MBH_FA
    return false;
}

}  // namespace mbh
