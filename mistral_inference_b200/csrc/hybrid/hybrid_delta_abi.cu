// C ABI of the gated delta rule (hybrid_delta.cuh); declarations and conventions: include/mistral_b200_hybrid.h.
#include "hybrid_delta.cuh"
#include "hybrid_error.h"
#include "../../../include/mistral_b200_hybrid.h"

using namespace mbh;

static int fail(cudaError_t e, const char* what) { return mbh_fail(e, what); }
static int bad(const char* what) { return mbh_bad(what); }

// key size -> lanes per state column and float4 per lane; tokens per shared-memory tile
template <int LANES, int RPL4, int C, int TB> static void run_delta_scan(const DeltaArgs& a, cudaStream_t st) {
    constexpr int NT = 128, COLS = C * NT / LANES;
    delta_scan_kernel<LANES, RPL4, C, TB, NT, (TB > 4 ? 4 : TB)><<<dim3((unsigned)(a.B * a.H), (unsigned)((a.e + COLS - 1) / COLS)), NT, 0, st>>>(a);
}
template <int C> static void run_delta_scan_keys(const DeltaArgs& a, cudaStream_t st) {
    if (a.d <= 32) run_delta_scan<8, 1, C, 16>(a, st);
    else if (a.d <= 64) run_delta_scan<8, 2, C, 16>(a, st);
    else if (a.d <= 128) run_delta_scan<8, 4, C, 8>(a, st);
    else if (a.d <= 256) run_delta_scan<8, 8, C, 4>(a, st);
    else run_delta_scan<32, 8, C, 1>(a, st);
}
// one column per lane group while that is about a CTA per SM (the scan then waits on its own reductions), two columns beyond it (shared
// memory reads are the limit, and each serves both)
static cudaError_t launch_delta_scan(const DeltaArgs& a, cudaStream_t st) {
    if ((int64_t)a.B * a.H * ((a.e + 15) / 16) <= 192) run_delta_scan_keys<1>(a, st);
    else run_delta_scan_keys<2>(a, st);
    return cudaGetLastError();
}
template <typename T, int TAPS> static void launch_delta_prep_tiled(const DeltaArgs& a, cudaStream_t st) {
    const dim3 grid((unsigned)((a.T + DP_WARPS * DP_TILE - 1) / (DP_WARPS * DP_TILE)), (unsigned)(a.G + a.H));
    if (a.d <= 128) delta_prep_tiled_kernel<T, TAPS, 1><<<grid, DP_WARPS * 32, 0, st>>>(a);
    else delta_prep_tiled_kernel<T, TAPS, 2><<<grid, DP_WARPS * 32, 0, st>>>(a);
}
template <typename T> static cudaError_t launch_delta_prep(const DeltaArgs& a, cudaStream_t st) {
    const bool tiled = a.taps <= 4 && a.d <= 256 && a.d % 4 == 0 && a.e % 4 == 0 && a.y_pitch % 4 == 0 && a.G + a.H <= 65535 &&
                       (reinterpret_cast<uintptr_t>(a.y) | reinterpret_cast<uintptr_t>(a.cstate) | reinterpret_cast<uintptr_t>(a.qk) | reinterpret_cast<uintptr_t>(a.v)) % 16 == 0;
    if (tiled) {
        if (a.taps == 1) launch_delta_prep_tiled<T, 1>(a, st);
        else if (a.taps == 2) launch_delta_prep_tiled<T, 2>(a, st);
        else if (a.taps == 3) launch_delta_prep_tiled<T, 3>(a, st);
        else launch_delta_prep_tiled<T, 4>(a, st);
    } else {
        const unsigned tiles = (unsigned)((a.T + DP_WARPS - 1) / DP_WARPS), units = (unsigned)(a.G + a.H);
        const dim3 grid(tiles, units < 65535u ? units : 65535u);
        if (a.d <= 64) delta_prep_kernel<T, 2><<<grid, DP_WARPS * 32, 0, st>>>(a);
        else if (a.d <= 128) delta_prep_kernel<T, 4><<<grid, DP_WARPS * 32, 0, st>>>(a);
        else if (a.d <= 256) delta_prep_kernel<T, 8><<<grid, DP_WARPS * 32, 0, st>>>(a);
        else delta_prep_kernel<T, 32><<<grid, DP_WARPS * 32, 0, st>>>(a);
    }
    if (a.taps > 1) delta_conv_state_kernel<T><<<dim3((unsigned)a.B, (unsigned)((2 * a.G * a.d + a.H * a.e + 255) / 256)), 256, 0, st>>>(a);
    return cudaGetLastError();
}
template <typename T, int LANES, int RPL4, int MIN_CTAS> static cudaError_t run_delta_step(DeltaArgs a, cudaStream_t st) {
    constexpr int D = DeltaColumn<LANES, RPL4>::DMAX;
    const size_t small = sizeof(float) * (3 * (size_t)D + 3 * (size_t)a.e + a.ra + a.rg), slices = sizeof(T) * ((size_t)a.d * a.ra + (size_t)a.e * a.rg);
    // the head's slices of the second projections are staged when they are made of 16-byte pieces and two CTAs still fit on an SM
    a.stage = a.ra * sizeof(T) % 16 == 0 && a.rg * sizeof(T) % 16 == 0 && small + slices + 16 <= 100 * 1024 &&
              (reinterpret_cast<uintptr_t>(a.w_a2) | reinterpret_cast<uintptr_t>(a.w_g2)) % 16 == 0;
    const size_t smem = small + (a.stage ? slices + 16 : 0);
    if (smem > 220 * 1024) return cudaErrorInvalidValue;
    cudaError_t e = cudaFuncSetAttribute(delta_step_kernel<T, LANES, RPL4, MIN_CTAS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e) return e;
    delta_step_kernel<T, LANES, RPL4, MIN_CTAS><<<(unsigned)(a.B * a.H), DT_THREADS, smem, st>>>(a);
    return cudaGetLastError();
}
template <typename T> static cudaError_t launch_delta_step(const DeltaArgs& a, cudaStream_t st) {
    if (a.d <= 32) return run_delta_step<T, 8, 1, 2>(a, st);
    if (a.d <= 64) return run_delta_step<T, 8, 2, 2>(a, st);
    if (a.d <= 128) return run_delta_step<T, 8, 4, 2>(a, st);
    if (a.d <= 256) return run_delta_step<T, 8, 8, 1>(a, st);
    return run_delta_step<T, 32, 8, 1>(a, st);
}

extern "C" {

int mbh_delta_prep(const void* y, int64_t y_pitch, const void* conv, int64_t taps, void* cstate, const void* positions, const void* q_start, const void* seqpos,
                   const void* slots, void* qk, void* kq, void* v, void* beta, int64_t T, int64_t B, int64_t H, int64_t G, int64_t d, int64_t e, int dt,
                   void* stream) {
    if (T == 0 || B == 0) return 0;
    if (d < 1 || d > 1024 || e < 1 || G < 1 || H % G) return bad("mbh_delta_prep: key size 1 .. 1024, heads a multiple of key heads");
    if (taps < 1) return bad("mbh_delta_prep: at least one tap");
    DeltaArgs a{};
    a.y = y; a.y_pitch = (int)y_pitch; a.conv = conv; a.taps = (int)taps; a.cstate = (float*)cstate;
    a.positions = (const int*)positions; a.q_start = (const int*)q_start; a.seqpos = (const int*)seqpos; a.slots = (const int*)slots;
    a.T = (int)T; a.B = (int)B; a.H = (int)H; a.G = (int)G; a.d = (int)d; a.e = (int)e;
    a.qk = (float*)qk; a.kq = (float*)kq; a.v = (float*)v; a.beta = (float*)beta;
    cudaError_t err = cudaSuccess;
    DISPATCH(dt, err = launch_delta_prep<ST>(a, (cudaStream_t)stream));
    return err ? fail(err, "mbh_delta_prep") : 0;
}

int mbh_delta_scan(const void* qk, const void* kq, const void* v, const void* beta, const void* g, void* state, const void* q_start, const void* seqpos,
                   const void* slots, void* o32, int64_t B, int64_t H, int64_t G, int64_t d, int64_t e, void* stream) {
    if (B == 0) return 0;
    if (d < 1 || d > 1024 || e < 1 || G < 1 || H % G) return bad("mbh_delta_scan: key size 1 .. 1024, heads a multiple of key heads");
    DeltaArgs a{};
    a.q_start = (const int*)q_start; a.seqpos = (const int*)seqpos; a.slots = (const int*)slots; a.state = (float*)state;
    a.B = (int)B; a.H = (int)H; a.G = (int)G; a.d = (int)d; a.e = (int)e;
    a.qk = (float*)const_cast<void*>(qk); a.kq = (float*)const_cast<void*>(kq); a.v = (float*)const_cast<void*>(v); a.beta = (float*)const_cast<void*>(beta);
    a.g = (const float*)g; a.o = (float*)o32;
    cudaError_t err = launch_delta_scan(a, (cudaStream_t)stream);
    return err ? fail(err, "mbh_delta_scan") : 0;
}

int mbh_delta_step(const void* y, int64_t y_pitch, int64_t ra, int64_t rg, const void* conv, int64_t taps, void* cstate, void* state, const void* w_a2,
                   const void* dt_bias, const void* a_log, const void* w_g2, const void* norm, const void* positions, const void* seqpos, const void* slots,
                   void* out, int64_t B, int64_t H, int64_t G, int64_t d, int64_t e, float eps, int dt, void* stream) {
    if (B == 0) return 0;
    if (d < 1 || d > 1024 || e < 1 || G < 1 || H % G) return bad("mbh_delta_step: key size 1 .. 1024, heads a multiple of key heads");
    if (taps < 1) return bad("mbh_delta_step: at least one tap");
    DeltaArgs a{};
    a.y = y; a.y_pitch = (int)y_pitch; a.ra = (int)ra; a.rg = (int)rg; a.conv = conv; a.taps = (int)taps; a.cstate = (float*)cstate; a.state = (float*)state;
    a.w_a2 = w_a2; a.dt_bias = dt_bias; a.a_log = a_log; a.w_g2 = w_g2; a.norm = norm;
    a.positions = (const int*)positions; a.seqpos = (const int*)seqpos; a.slots = (const int*)slots;
    a.T = (int)B; a.B = (int)B; a.H = (int)H; a.G = (int)G; a.d = (int)d; a.e = (int)e; a.eps = eps; a.out = out;
    cudaError_t err = cudaSuccess;
    DISPATCH(dt, err = launch_delta_step<ST>(a, (cudaStream_t)stream));
    return err ? fail(err, "mbh_delta_step") : 0;
}

}  // extern "C"
