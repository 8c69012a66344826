// The error text of libmb200_hybrid.so's calls and the choice of storage type, shared by its translation units.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>

int mbh_fail(cudaError_t e, const char* what);  // leaves "what: <text of e>", returns e
int mbh_bad(const char* what);                  // leaves what, returns -1

#define DISPATCH(dt, ...)                                   \
    do {                                                    \
        if ((dt) == 0) { using ST = __nv_bfloat16; __VA_ARGS__; }     \
        else if ((dt) == 1) { using ST = float; __VA_ARGS__; } \
        else return mbh_bad("dt must be 0 (bf16) or 1 (fp32)"); \
    } while (0)
