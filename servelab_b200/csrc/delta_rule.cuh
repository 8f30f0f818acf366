// What the kernels of the delta rule share: their argument block and its check (the recurrence itself
// is described in delta_rule.cu).
#pragma once

#include "common.cuh"

#define DR_MAX_D 256

struct DeltaRuleArgs {
    const void* proj; int ld;
    int r_off, k_off, v_off, a_off;
    int H, D, Dv;
    const float* a_bias;                     // [H * D]
    const float* gate_z; int ld_gate; float decay_coef; float unit_eps;
    const int* cu_q; const int* state_slots;
    float* state; int num_slots; long long state_stride;
    float* out; int ldo;                     // [T][H * Dv] float32 (not with out_t)
    // with out_t: every head's result divided by its root mean square, times norm_w [H * Dv], times
    // sigmoid of the gate columns of proj, in the compute type
    void* out_t; int ldt; int g_off; const float* norm_w; float norm_eps;
};

__device__ __forceinline__ float dr_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }

static inline int dr_check(const DeltaRuleArgs& a) {
    if (a.H <= 0 || a.D <= 0 || a.Dv <= 0 || a.num_slots <= 0 || a.state == nullptr || a.gate_z == nullptr ||
        a.ld_gate < a.H * a.D || a.a_bias == nullptr || a.state_stride < (long long)a.H * a.D * a.Dv ||
        !(a.decay_coef >= 0.f) || (a.out == nullptr) == (a.out_t == nullptr) ||
        (a.out_t != nullptr && a.norm_w == nullptr))
        return SLB_ERR_BAD_ARG;
    if (a.D > DR_MAX_D || a.H > 65535) return SLB_ERR_TOO_LARGE;
    return 0;
}
