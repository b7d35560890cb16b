// The gates of the matrix memory, shared by its two forms.
#pragma once

#include "api.h"
#include "common.cuh"

#define MM_COLS 32             // columns of the state a block of the scan owns; n and m are kept once for so many
#define MM_MAX_PREFETCH 2      // raw values of q and of k a thread of the scan brings for the next token
#define MM_LOG2E 1.4426950408889634f

static inline int mm_copies(int vdim) { return (vdim + MM_COLS - 1) / MM_COLS; }
int rdl_check_matrix_memory_args(const MatrixMemoryArgs* a, const char* who);

// logarithms to base two
__device__ __forceinline__ float mm_input_gate(float x, float bias, float cap) { return cap * tanhf((x + bias) / cap) * MM_LOG2E; }
__device__ __forceinline__ float mm_forget_gate(float x, float bias, float cap) {
    const float z = cap * tanhf((x + bias) / cap);
    return (fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * MM_LOG2E;
}
