// Linear attention by a delta rule with a decay per key channel, over a per-request state S (D x Dv
// float32 a head, kept in a state slot):
//
//     u_t = k_t / sqrt(sum k_t^2 + eps)
//     S_t = diag(w_t) S_{t-1} - (a_t u_t) (u_t^T S_{t-1}) + k_t v_t^T,     o_t = S_t^T r_t
//
// (both terms of the update read the old state), with w_t = exp(-coef sigmoid(z_t)) and
// a_t = sigmoid(x_t + b) per head and key channel; z arrives in float32, r, k, v, x are columns of one
// projected row per token.  Everything after the load is float32.
//
// Token by token (`delta_rule_kernel`): steps of single tokens, short portions, the 32-bit path.
// Chunked (delta_rule_chunk.cu): longer portions.  Both can cut a request anywhere.
#include "delta_rule.cuh"

// ------------------------------------------------------------------ token by token
// Row of S that element i (of R = 4 * groups) of part p holds: groups of four rows are dealt out to the
// eight parts in turn, so that the parts of a warp read neighbouring 16-byte pieces of a staged row.
//
// Since o_t = S_t^T r = (diag(w) S_{t-1})^T r - (sum r a u) (S_{t-1}^T u) + (sum r k) v, one pass over
// the old state gives both sums that a token needs, and the parts add them up once.
//
// A warp owns 4 CV value columns: lane = 8 * column group + part; a thread keeps R rows of CV columns
// in registers.
#define DR_TT 8
#define DR_MAX_WARPS 16

template <typename T, int R, int CV>
__global__ void __launch_bounds__(DR_MAX_WARPS * 32, 1) delta_rule_kernel(const DeltaRuleArgs a) {
    extern __shared__ __align__(16) float dr_smem[];
    pdl_wait();
    pdl_launch_dependents();
    const int s = blockIdx.x, h = blockIdx.y;
    const int q0 = a.cu_q[s];
    const int qlen = a.cu_q[s + 1] - q0;
    if (qlen <= 0) return;
    const int slot = a.state_slots[s];
    if (slot < 0 || slot >= a.num_slots) return;
    const int D = a.D, Dv = a.Dv;
    constexpr int LD = R * 8;
    const int nwarps = blockDim.x >> 5;
    const int ncols = nwarps * 4 * CV;                     // value columns of this block
    const int e0 = blockIdx.z * ncols;
    float* us = dr_smem;                                   // [DR_TT][LD]: unit key
    float* rs = us + DR_TT * LD;                           // r times the decay
    float* ws = rs + DR_TT * LD;                           // decay
    float* as = ws + DR_TT * LD;                           // removal rate times unit key
    float* ks = as + DR_TT * LD;
    float* vs = ks + DR_TT * LD;                           // [DR_TT][ncols]
    float* os = vs + DR_TT * ncols;                        // [DR_TT][ncols]
    float* cs = os + DR_TT * ncols;                        // [DR_TT][2]: sum r a u, sum r k
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int p = lane & 7, cg = lane >> 3;
    const int lcol = (warp * 4 + cg) * CV, col = e0 + lcol;
    float* S = a.state + (size_t)slot * a.state_stride + (size_t)h * D * Dv;
    const bool wide = CV == 4 && (Dv & 3) == 0 && col + CV <= Dv && ((uintptr_t)S & 15) == 0;
    float st[R][CV];
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int d = ((i >> 2) * 8 + p) * 4 + (i & 3);
#pragma unroll
        for (int c = 0; c < CV; ++c) st[i][c] = 0.f;
        if (d < D) {
            if (wide) {
                if constexpr (CV == 4) {
                    const float4 x = *reinterpret_cast<const float4*>(S + (size_t)d * Dv + col);
                    st[i][0] = x.x; st[i][1] = x.y; st[i][2] = x.z; st[i][3] = x.w;
                }
            } else {
#pragma unroll
                for (int c = 0; c < CV; ++c)
                    if (col + c < Dv) st[i][c] = S[(size_t)d * Dv + col + c];
            }
        }
    }
    const T* proj = reinterpret_cast<const T*>(a.proj);
    for (int t0 = 0; t0 < qlen; t0 += DR_TT) {
        const int n = min(DR_TT, qlen - t0);
        __syncthreads();                                   // (the previous tile's rows have been read)
        for (int j = warp; j < n; j += nwarps) {           // a warp prepares a token's rows
            const T* row = proj + (size_t)(q0 + t0 + j) * a.ld;
            const float* zr = a.gate_z + (size_t)(q0 + t0 + j) * a.ld_gate + h * D;
            float ss = 0.f;
            for (int d = lane; d < D; d += 32) {
                const float k = to_float(row[a.k_off + h * D + d]);
                ss = fmaf(k, k, ss);
            }
            ss = warp_sum(ss);
            const float inv = 1.0f / sqrtf(ss + a.unit_eps);
            float c1 = 0.f, c2 = 0.f;
            for (int d = lane; d < LD; d += 32) {
                float u = 0.f, rw = 0.f, w = 0.f, au = 0.f, k = 0.f;
                if (d < D) {
                    k = to_float(row[a.k_off + h * D + d]);
                    const float r = to_float(row[a.r_off + h * D + d]);
                    w = decay_exp(-a.decay_coef * dr_sigmoid(zr[d]));
                    u = k * inv;
                    au = dr_sigmoid(to_float(row[a.a_off + h * D + d]) + a.a_bias[h * D + d]) * u;
                    rw = r * w;
                    c1 = fmaf(r, au, c1);
                    c2 = fmaf(r, k, c2);
                }
                us[j * LD + d] = u; rs[j * LD + d] = rw; ws[j * LD + d] = w; as[j * LD + d] = au; ks[j * LD + d] = k;
            }
            c1 = warp_sum(c1);
            c2 = warp_sum(c2);
            if (lane == 0) { cs[2 * j] = c1; cs[2 * j + 1] = c2; }
            for (int c = lane; c < ncols; c += 32)
                vs[j * ncols + c] = e0 + c < Dv ? to_float(row[a.v_off + h * Dv + e0 + c]) : 0.f;
        }
        __syncthreads();
        for (int j = 0; j < n; ++j) {
            float seen[CV], y[CV];
#pragma unroll
            for (int c = 0; c < CV; ++c) seen[c] = y[c] = 0.f;
#pragma unroll
            for (int g = 0; g < R / 4; ++g) {
                const int at = j * LD + (g * 8 + p) * 4;
                const float4 u4 = *reinterpret_cast<const float4*>(us + at);
                const float4 r4 = *reinterpret_cast<const float4*>(rs + at);
                const float uu[4] = {u4.x, u4.y, u4.z, u4.w}, rr[4] = {r4.x, r4.y, r4.z, r4.w};
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int c = 0; c < CV; ++c) {
                        seen[c] = fmaf(uu[i], st[4 * g + i][c], seen[c]);
                        y[c] = fmaf(rr[i], st[4 * g + i][c], y[c]);
                    }
            }
#pragma unroll
            for (int o = 1; o < 8; o <<= 1)
#pragma unroll
                for (int c = 0; c < CV; ++c) {
                    seen[c] += __shfl_xor_sync(0xffffffffu, seen[c], o);
                    y[c] += __shfl_xor_sync(0xffffffffu, y[c], o);
                }
            float v[CV];
#pragma unroll
            for (int c = 0; c < CV; ++c) v[c] = vs[j * ncols + lcol + c];
            if (p == 0) {
                const float c1 = cs[2 * j], c2 = cs[2 * j + 1];
#pragma unroll
                for (int c = 0; c < CV; ++c) os[j * ncols + lcol + c] = fmaf(c2, v[c], fmaf(-c1, seen[c], y[c]));
            }
#pragma unroll
            for (int g = 0; g < R / 4; ++g) {
                const int at = j * LD + (g * 8 + p) * 4;
                const float4 w4 = *reinterpret_cast<const float4*>(ws + at);
                const float4 a4 = *reinterpret_cast<const float4*>(as + at);
                const float4 k4 = *reinterpret_cast<const float4*>(ks + at);
                const float ww[4] = {w4.x, w4.y, w4.z, w4.w}, aa[4] = {a4.x, a4.y, a4.z, a4.w};
                const float kk[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int c = 0; c < CV; ++c)
                        st[4 * g + i][c] = fmaf(ww[i], st[4 * g + i][c], fmaf(-aa[i], seen[c], kk[i] * v[c]));
            }
        }
        __syncthreads();
        if (a.out_t != nullptr) {                          // (the block holds every value column of the head)
            T* out = reinterpret_cast<T*>(a.out_t);
            for (int j = warp; j < n; j += nwarps) {
                const size_t t = q0 + t0 + j;
                float ss = 0.f;
                for (int c = lane; c < Dv; c += 32) ss = fmaf(os[j * ncols + c], os[j * ncols + c], ss);
                ss = warp_sum(ss);
                const float rstd = 1.0f / sqrtf(ss / (float)Dv + a.norm_eps);
                for (int c = lane; c < Dv; c += 32) {
                    const float g = to_float(proj[t * a.ld + a.g_off + h * Dv + c]);
                    out[t * a.ldt + h * Dv + c] =
                        from_float<T>(os[j * ncols + c] * rstd * a.norm_w[h * Dv + c] * dr_sigmoid(g));
                }
            }
        } else {
            for (int idx = tid; idx < n * ncols; idx += blockDim.x) {
                const int j = idx / ncols, c = idx - j * ncols;
                if (e0 + c < Dv) a.out[(size_t)(q0 + t0 + j) * a.ldo + h * Dv + e0 + c] = os[idx];
            }
        }
    }
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int d = ((i >> 2) * 8 + p) * 4 + (i & 3);
        if (d < D) {
            if (wide) {
                if constexpr (CV == 4)
                    *reinterpret_cast<float4*>(S + (size_t)d * Dv + col) =
                        make_float4(st[i][0], st[i][1], st[i][2], st[i][3]);
            } else {
#pragma unroll
                for (int c = 0; c < CV; ++c)
                    if (col + c < Dv) S[(size_t)d * Dv + col + c] = st[i][c];
            }
        }
    }
}

// rows a thread holds and columns a thread for key size D, and the warps (of 4 CV columns) for Dv columns
static void dr_shape(int D, int Dv, int& R, int& CV, int& warps) {
    R = D <= 32 ? 4 : D <= 64 ? 8 : D <= 128 ? 16 : 32;
    CV = R == 32 ? 2 : 4;
    warps = (Dv + 4 * CV - 1) / (4 * CV);
}

template <typename T, int R, int CV>
static int launch_delta_rule_rc(const DeltaRuleArgs& a, int num_seqs, int warps, int z, cudaStream_t st) {
    const size_t smem = ((size_t)5 * DR_TT * R * 8 + 2 * (size_t)DR_TT * warps * 4 * CV + 2 * DR_TT) * sizeof(float);
    constexpr size_t MAXS = ((size_t)5 * DR_TT * R * 8 + 2 * (size_t)DR_TT * DR_MAX_WARPS * 4 * CV + 2 * DR_TT) * sizeof(float);
    static unsigned long long configured = 0;
    const int rc = slb_configure(&configured, delta_rule_kernel<T, R, CV>, MAXS);
    if (rc != 0) return rc;
    return slb_launch(delta_rule_kernel<T, R, CV>, dim3(num_seqs, a.H, z), dim3(warps * 32), smem, st, a);
}

template <typename T>
static int launch_delta_rule(const DeltaRuleArgs& a, int num_seqs, cudaStream_t st) {
    if (num_seqs <= 0) return 0;
    const int rc = dr_check(a);
    if (rc != 0) return rc;
    int R, CV, warps;
    dr_shape(a.D, a.Dv, R, CV, warps);
    const int z = (warps + DR_MAX_WARPS - 1) / DR_MAX_WARPS;
    if (z > 1 && a.out_t != nullptr) return SLB_ERR_BAD_ARG;
    if (z > 1) warps = DR_MAX_WARPS;
    if (R == 4) return launch_delta_rule_rc<T, 4, 4>(a, num_seqs, warps, z, st);
    if (R == 8) return launch_delta_rule_rc<T, 8, 4>(a, num_seqs, warps, z, st);
    if (R == 16) return launch_delta_rule_rc<T, 16, 4>(a, num_seqs, warps, z, st);
    return launch_delta_rule_rc<T, 32, 2>(a, num_seqs, warps, z, st);
}

extern "C" {
int slb_delta_rule_max_dim() { return DR_MAX_D; }
// 1 if the token-by-token kernel's block holds every value column of a head (the fused norm and gate)
int slb_delta_rule_fuses(int D, int Dv) {
    int R, CV, warps;
    if (D <= 0 || D > DR_MAX_D || Dv <= 0) return 0;
    dr_shape(D, Dv, R, CV, warps);
    return warps <= DR_MAX_WARPS;
}
int slb_delta_rule_f32(const DeltaRuleArgs* a, int num_seqs, cudaStream_t st) {
    return launch_delta_rule<float>(*a, num_seqs, st);
}
int slb_delta_rule_bf16(const DeltaRuleArgs* a, int num_seqs, cudaStream_t st) {
    return launch_delta_rule<bf16>(*a, num_seqs, st);
}
}
