// What the kernels of the selective state space share: their argument block, the step size and the
// logarithm of the decay.
#pragma once

#include "common.cuh"

struct StateSpaceArgs {
    const void* u; int ld;         // [T][...]: x [H * P] | B [G * N] | C [G * N], convolved and activated
    int x_off, b_off, c_off;
    int H, P, N, G;                // heads, value size, state size, groups (head h reads group h / (H / G))
    const float* dt; int ld_dt;    // [T][H]: logits of the step sizes
    const float* dt_bias;          // [H]
    const float* rate;             // [H], positive: exp(A_log)
    const float* skip;             // [H]: D
    const int* cu_q; const int* state_slots;
    float* state; int num_slots; long long state_stride;     // a record: [H][N][P] float32
    float* out; int ldo;           // [T][H * P] float32
};

// softplus(z) = log(1 + e^z)
__device__ __forceinline__ float ss_step(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
