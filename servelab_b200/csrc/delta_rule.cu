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
// Chunked (`delta_chunk_*`): longer portions.  Both can cut a request anywhere.
#include "mma_util.cuh"

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
#define DR_MAX_D 256
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

static int dr_check(const DeltaRuleArgs& a) {
    if (a.H <= 0 || a.D <= 0 || a.Dv <= 0 || a.num_slots <= 0 || a.state == nullptr || a.gate_z == nullptr ||
        a.ld_gate < a.H * a.D || a.a_bias == nullptr || a.state_stride < (long long)a.H * a.D * a.Dv ||
        !(a.decay_coef >= 0.f) || (a.out == nullptr) == (a.out_t == nullptr) ||
        (a.out_t != nullptr && a.norm_w == nullptr))
        return SLB_ERR_BAD_ARG;
    if (a.D > DR_MAX_D || a.H > 65535) return SLB_ERR_TOO_LARGE;
    return 0;
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

// ------------------------------------------------------------------ in chunks
// A chunk of C = 32 tokens with entering state S.  L_t: sum of log w up to and including token t
// (per channel), G_t = e^(L_t).  With seen_t = u_t^T S_{t-1} and b_t = a_t u_t,
//
//     S_t    = G_t S + sum_{j <= t} (G_t / G_j) (k_j v_j^T - b_j seen_j^T)
//     seen_t = (u_t G_{t-1})^T S + sum_{j < t} (N[t][j] v_j - M[t][j] seen_j),
//              N[t][j] = sum_d u_t G_{t-1} k_j / G_j,   M[t][j] = sum_d u_t G_{t-1} b_j / G_j
//     o_t    = (r_t G_t)^T S + sum_{j <= t} (P[t][j] v_j - Q[t][j] seen_j),
//              P[t][j] = sum_d r_t G_t k_j / G_j,       Q[t][j] = sum_d r_t G_t b_j / G_j
//
// so with the unit lower triangle I + M solved for its right-hand sides once,
//
//     seen = X S + Y v,   X = (I + M)^-1 (u G_{t-1}),   Y = (I + M)^-1 N.
//
// The factors 1 / G_j are formed alone: a step's log decay is at least -coef, so over a chunk they stay
// below e^(32 coef) (the launcher takes coef <= 2), and every product of two factors has the relative
// error of its factors.  Two launches: `prep` per (chunk, head) leaves X, Y, P, Q, the decayed rows
// r_t G_t, k_j G_C / G_j, b_j G_C / G_j and G_C in a work buffer; `scan` walks a request's chunks with 16
// value columns of the state a block.  float32 on the CUDA cores throughout.
#define DC_C 32
#define DC_EV 16

struct DeltaChunkArgs {
    DeltaRuleArgs a;
    const int* tile_seq; const int* tile_row0; int num_tiles;
    float* work;                             // [num_tiles][H][dc_floats(D)]
};

// a (chunk, head)'s record: X, R, K, B as [C][Dp], then Y, P, Q as [C][C], then G_C [Dp]
__host__ __device__ constexpr int dc_pad(int D) { return (D + 3) & ~3; }
__host__ __device__ constexpr size_t dc_floats(int D) {
    return (size_t)4 * DC_C * dc_pad(D) + 3 * DC_C * DC_C + dc_pad(D);
}

__device__ __forceinline__ bool dc_tile(const DeltaChunkArgs& c, int tile, int& t0, int& n) {
    const int s = c.tile_seq[tile];
    const int q0 = c.a.cu_q[s], row0 = c.tile_row0[tile];
    n = min(DC_C, c.a.cu_q[s + 1] - q0 - row0);
    t0 = q0 + row0;
    return n > 0;
}

template <typename T>
__global__ void __launch_bounds__(256) delta_chunk_prep_kernel(const DeltaChunkArgs c) {
    extern __shared__ __align__(16) float dc_smem[];
    pdl_wait();
    pdl_launch_dependents();
    const DeltaRuleArgs& a = c.a;
    const int tile = blockIdx.x, h = blockIdx.y;
    int t0, n;
    if (!dc_tile(c, tile, t0, n)) return;
    const int D = a.D, Dp = dc_pad(D), LD = Dp + 4;
    float* Ls = dc_smem;                         // [C][LD]: log decays, then their running sums
    float* Rs = Ls + DC_C * LD;                  // r_t G_t          (rows 0..31 of the left operand)
    float* Us = Rs + DC_C * LD;                  // u_t G_{t-1}      (rows 32..63)
    float* Ks = Us + DC_C * LD;                  // k_j / G_j        (rows 0..31 of the right operand)
    float* Bs = Ks + DC_C * LD;                  // a_j u_j / G_j    (rows 32..63)
    float* Gm = Bs + DC_C * LD;                  // [64][68]: the products of the two operands
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const T* proj = reinterpret_cast<const T*>(a.proj);
    for (int idx = tid; idx < DC_C * Dp; idx += blockDim.x) {
        const int j = idx / Dp, d = idx - j * Dp;
        float l = 0.f;
        if (j < n && d < D) l = -a.decay_coef * dr_sigmoid(a.gate_z[(size_t)(t0 + j) * a.ld_gate + h * D + d]);
        Ls[j * LD + d] = l;
    }
    __syncthreads();
    for (int d = tid; d < Dp; d += blockDim.x) {
        float run = 0.f;
        for (int j = 0; j < DC_C; ++j) {
            run += Ls[j * LD + d];
            Ls[j * LD + d] = run;                // (beyond the chunk's tokens the sum stays what it is)
        }
    }
    __syncthreads();
    float* rec = c.work + ((size_t)tile * a.H + h) * dc_floats(D);
    float* gX = rec, *gR = gX + DC_C * Dp, *gK = gR + DC_C * Dp, *gB = gK + DC_C * Dp;
    float* gY = gB + DC_C * Dp, *gP = gY + DC_C * DC_C, *gQ = gP + DC_C * DC_C, *gG = gQ + DC_C * DC_C;
    for (int j = warp; j < DC_C; j += 8) {
        if (j >= n) {
            for (int d = lane; d < Dp; d += 32) {
                Rs[j * LD + d] = Us[j * LD + d] = Ks[j * LD + d] = Bs[j * LD + d] = 0.f;
                gR[j * Dp + d] = gK[j * Dp + d] = gB[j * Dp + d] = 0.f;
            }
            continue;
        }
        const T* row = proj + (size_t)(t0 + j) * a.ld;
        float ss = 0.f;
        for (int d = lane; d < D; d += 32) {
            const float k = to_float(row[a.k_off + h * D + d]);
            ss = fmaf(k, k, ss);
        }
        ss = warp_sum(ss);
        const float inv = 1.0f / sqrtf(ss + a.unit_eps);
        for (int d = lane; d < Dp; d += 32) {
            float rg = 0.f, ug = 0.f, kg = 0.f, bg = 0.f, ke = 0.f, be = 0.f;
            if (d < D) {
                const float L = Ls[j * LD + d], Lp = j > 0 ? Ls[(j - 1) * LD + d] : 0.f, Le = Ls[(DC_C - 1) * LD + d];
                const float k = to_float(row[a.k_off + h * D + d]), r = to_float(row[a.r_off + h * D + d]);
                const float u = k * inv;
                const float b = dr_sigmoid(to_float(row[a.a_off + h * D + d]) + a.a_bias[h * D + d]) * u;
                const float up = expf(-L), rest = expf(Le - L);
                rg = r * expf(L);
                ug = u * expf(Lp);
                kg = k * up;
                bg = b * up;
                ke = k * rest;
                be = b * rest;
            }
            Rs[j * LD + d] = rg; Us[j * LD + d] = ug; Ks[j * LD + d] = kg; Bs[j * LD + d] = bg;
            gR[j * Dp + d] = rg; gK[j * Dp + d] = ke; gB[j * Dp + d] = be;
        }
    }
    for (int d = tid; d < Dp; d += blockDim.x) gG[d] = decay_exp(Ls[(DC_C - 1) * LD + d]);
    __syncthreads();
    // the four score matrices as one 64 x 64 product; thread (ty, tx): rows ty + 16 i, columns tx + 16 j
    {
        const int tx = tid & 15, ty = tid >> 4;
        float acc[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
        const float* A0 = Rs + ty * LD;          // (Us follows Rs, Bs follows Ks: one 64-row operand each)
        const float* B0 = Ks + tx * LD;
        for (int d = 0; d < Dp; d += 4) {
            float4 x[4], y[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                x[i] = *reinterpret_cast<const float4*>(A0 + i * 16 * LD + d);
                y[i] = *reinterpret_cast<const float4*>(B0 + i * 16 * LD + d);
            }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    acc[i][j] = fmaf(x[i].x, y[j].x, acc[i][j]);
                    acc[i][j] = fmaf(x[i].y, y[j].y, acc[i][j]);
                    acc[i][j] = fmaf(x[i].z, y[j].z, acc[i][j]);
                    acc[i][j] = fmaf(x[i].w, y[j].w, acc[i][j]);
                }
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int r = ty + 16 * i, q = tx + 16 * j;
                const int t = r & 31, jj = q & 31;
                const bool keep = r < 32 ? jj <= t : jj < t;
                const float v = keep ? acc[i][j] : 0.f;
                Gm[r * 68 + q] = v;
                if (r < 32) (q < 32 ? gP : gQ)[t * DC_C + jj] = v;
            }
    }
    __syncthreads();
    // (I + M) z = rhs, a column a thread: the D columns of u G_{t-1} give X, the 32 of N give Y
    for (int col = tid; col < Dp + DC_C; col += blockDim.x) {
        float z[DC_C];
        const bool isX = col < Dp;
#pragma unroll
        for (int t = 0; t < DC_C; ++t) {
            float v = isX ? Us[t * LD + col] : Gm[(32 + t) * 68 + (col - Dp)];
            const float* m = Gm + (32 + t) * 68 + 32;
#pragma unroll
            for (int j4 = 0; j4 < (t + 3) / 4; ++j4) {     // (M is zero from column t on)
                const float4 m4 = *reinterpret_cast<const float4*>(m + 4 * j4);
                v = fmaf(-m4.x, z[4 * j4], v);
                if (4 * j4 + 1 < t) v = fmaf(-m4.y, z[4 * j4 + 1], v);
                if (4 * j4 + 2 < t) v = fmaf(-m4.z, z[4 * j4 + 2], v);
                if (4 * j4 + 3 < t) v = fmaf(-m4.w, z[4 * j4 + 3], v);
            }
            z[t] = v;
            if (isX) gX[t * Dp + col] = v;
            else gY[t * DC_C + col - Dp] = v;
        }
    }
}

// STAGES 2: the next chunk's record is fetched while this one is worked on.
template <typename T, int STAGES>
__global__ void __launch_bounds__(256) delta_chunk_scan_kernel(const DeltaChunkArgs c) {
    extern __shared__ __align__(16) float dc_smem[];
    __shared__ int first_s;
    pdl_wait();
    const DeltaRuleArgs& a = c.a;
    const int s = blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * DC_EV;
    const int q0 = a.cu_q[s];
    const int qlen = a.cu_q[s + 1] - q0;
    if (qlen <= 0) return;
    const int slot = a.state_slots[s];
    if (slot < 0 || slot >= a.num_slots) return;
    const int tid = threadIdx.x;
    if (tid == 0) first_s = c.num_tiles;
    __syncthreads();
    for (int i = tid; i < c.num_tiles; i += blockDim.x)     // a request's chunks are neighbours in the list, in order
        if (c.tile_seq[i] == s) { atomicMin(&first_s, i); break; }
    __syncthreads();
    const int first = first_s;
    const int count = (qlen + DC_C - 1) / DC_C;
    if (first + count > c.num_tiles) return;
    const int D = a.D, Dv = a.Dv, Dp = dc_pad(D), LD = Dp + 4;
    // a stage: X [C][LD], R [C][LD], K [C][Dp], B [C][Dp], Y, P, Q [C][C], G [Dp], V [C][EV]
    const int XR = 2 * DC_C * LD, KB = 2 * DC_C * Dp, YPQ = 3 * DC_C * DC_C;
    const int stage_floats = XR + KB + YPQ + Dp + DC_C * DC_EV;
    float* Ss = dc_smem;                                    // [Dp][EV]
    float* Sn = Ss + Dp * DC_EV;                            // [C][EV]: seen
    float* stages = Sn + DC_C * DC_EV;
    const T* proj = reinterpret_cast<const T*>(a.proj);
    float* gS = a.state + (size_t)slot * a.state_stride + (size_t)h * D * Dv;
    for (int idx = tid; idx < Dp * DC_EV; idx += blockDim.x) {
        const int d = idx / DC_EV, e = e0 + idx % DC_EV;
        Ss[idx] = d < D && e < Dv ? gS[(size_t)d * Dv + e] : 0.f;
    }
    const int dq = Dp / 4;
    auto fetch = [&](int k) {
        float* b = stages + (k % STAGES) * stage_floats;
        const float* rec = c.work + ((size_t)(first + k) * a.H + h) * dc_floats(D);
        for (int idx = tid; idx < 2 * DC_C * dq; idx += blockDim.x) {
            const int r = idx / dq, d4 = idx - r * dq;
            slb_mma::cp_async16(b + r * LD + d4 * 4, rec + r * Dp + d4 * 4, true);
        }
        const float* rest = rec + 2 * DC_C * Dp;
        float* dst = b + XR;
        const int quads = (KB + YPQ + Dp) / 4;
        for (int idx = tid; idx < quads; idx += blockDim.x) slb_mma::cp_async16(dst + idx * 4, rest + idx * 4, true);
        slb_mma::cp_async_commit();
        float* vs = b + XR + KB + YPQ + Dp;
        for (int idx = tid; idx < DC_C * DC_EV; idx += blockDim.x) {
            const int j = idx / DC_EV, e = e0 + idx % DC_EV;
            const int t = k * DC_C + j;
            vs[idx] = t < qlen && e < Dv ? to_float(proj[(size_t)(q0 + t) * a.ld + a.v_off + h * Dv + e]) : 0.f;
        }
    };
    if (STAGES == 2) fetch(0);
    const int cq = (tid & 3) * 4, row = tid >> 2;
    for (int k = 0; k < count; ++k) {
        if (STAGES == 2) {
            if (k + 1 < count) {
                fetch(k + 1);
                slb_mma::cp_async_wait<1>();
            } else {
                slb_mma::cp_async_wait<0>();
            }
        } else {
            fetch(k);
            slb_mma::cp_async_wait<0>();
        }
        __syncthreads();
        const float* b = stages + (k % STAGES) * stage_floats;
        const float* Kd = b + XR, *Bd = Kd + DC_C * Dp, *Ym = b + XR + KB, *Pm = Ym + DC_C * DC_C, *Qm = Pm + DC_C * DC_C;
        const float* G = b + XR + KB + YPQ, *V = G + Dp;
        // rows 0..31: X S (+ Y V = seen); rows 32..63: R S, the state's part of the outputs
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
#define DC_ROW(xv, s4)                                                                           \
        acc[0] = fmaf(xv, s4.x, acc[0]); acc[1] = fmaf(xv, s4.y, acc[1]);                          \
        acc[2] = fmaf(xv, s4.z, acc[2]); acc[3] = fmaf(xv, s4.w, acc[3]);
        const float* xr = b + row * LD;
#pragma unroll 4
        for (int d = 0; d < Dp; d += 4) {
            const float4 x4 = *reinterpret_cast<const float4*>(xr + d);
            const float4 s0 = *reinterpret_cast<const float4*>(Ss + d * DC_EV + cq);
            const float4 s1 = *reinterpret_cast<const float4*>(Ss + (d + 1) * DC_EV + cq);
            const float4 s2 = *reinterpret_cast<const float4*>(Ss + (d + 2) * DC_EV + cq);
            const float4 s3 = *reinterpret_cast<const float4*>(Ss + (d + 3) * DC_EV + cq);
            DC_ROW(x4.x, s0) DC_ROW(x4.y, s1) DC_ROW(x4.z, s2) DC_ROW(x4.w, s3)
        }
        {
            // both halves add their product with V: Y for the seen rows, P for the outputs
            const float* m = row < DC_C ? Ym + row * DC_C : Pm + (row - DC_C) * DC_C;
#pragma unroll 2
            for (int j = 0; j < DC_C; j += 4) {
                const float4 m4 = *reinterpret_cast<const float4*>(m + j);
                const float4 v0 = *reinterpret_cast<const float4*>(V + j * DC_EV + cq);
                const float4 v1 = *reinterpret_cast<const float4*>(V + (j + 1) * DC_EV + cq);
                const float4 v2 = *reinterpret_cast<const float4*>(V + (j + 2) * DC_EV + cq);
                const float4 v3 = *reinterpret_cast<const float4*>(V + (j + 3) * DC_EV + cq);
                DC_ROW(m4.x, v0) DC_ROW(m4.y, v1) DC_ROW(m4.z, v2) DC_ROW(m4.w, v3)
            }
        }
        if (row < DC_C) *reinterpret_cast<float4*>(Sn + row * DC_EV + cq) = make_float4(acc[0], acc[1], acc[2], acc[3]);
        __syncthreads();
        if (row >= DC_C) {
            const int t = row - DC_C;
            const float* m = Qm + t * DC_C;
#pragma unroll 2
            for (int j = 0; j < DC_C; j += 4) {
                const float4 m4 = *reinterpret_cast<const float4*>(m + j);
                const float4 v0 = *reinterpret_cast<const float4*>(Sn + j * DC_EV + cq);
                const float4 v1 = *reinterpret_cast<const float4*>(Sn + (j + 1) * DC_EV + cq);
                const float4 v2 = *reinterpret_cast<const float4*>(Sn + (j + 2) * DC_EV + cq);
                const float4 v3 = *reinterpret_cast<const float4*>(Sn + (j + 3) * DC_EV + cq);
                DC_ROW(-m4.x, v0) DC_ROW(-m4.y, v1) DC_ROW(-m4.z, v2) DC_ROW(-m4.w, v3)
            }
            const int tt = k * DC_C + t;
            if (tt < qlen) {
                float* o = a.out + (size_t)(q0 + tt) * a.ldo + h * Dv + e0 + cq;
                if ((Dv & 3) == 0 && (a.ldo & 3) == 0) {
                    if (e0 + cq < Dv) *reinterpret_cast<float4*>(o) = make_float4(acc[0], acc[1], acc[2], acc[3]);
                } else {
#pragma unroll
                    for (int i = 0; i < 4; ++i)
                        if (e0 + cq + i < Dv) o[i] = acc[i];
                }
            }
        }
#undef DC_ROW
        // S <- G S + K^T V - B^T seen: a thread two neighbouring rows of four columns at a time
        for (int d = row * 2; d < Dp; d += 128) {
            float4 s0 = *reinterpret_cast<const float4*>(Ss + d * DC_EV + cq);
            float4 s1 = *reinterpret_cast<const float4*>(Ss + (d + 1) * DC_EV + cq);
            const float g0 = G[d], g1 = G[d + 1];
            s0.x *= g0; s0.y *= g0; s0.z *= g0; s0.w *= g0;
            s1.x *= g1; s1.y *= g1; s1.z *= g1; s1.w *= g1;
#pragma unroll 4
            for (int j = 0; j < DC_C; ++j) {
                const float2 k2 = *reinterpret_cast<const float2*>(Kd + j * Dp + d);
                const float2 b2 = *reinterpret_cast<const float2*>(Bd + j * Dp + d);
                const float4 v = *reinterpret_cast<const float4*>(V + j * DC_EV + cq);
                const float4 q = *reinterpret_cast<const float4*>(Sn + j * DC_EV + cq);
                s0.x = fmaf(k2.x, v.x, fmaf(-b2.x, q.x, s0.x));
                s0.y = fmaf(k2.x, v.y, fmaf(-b2.x, q.y, s0.y));
                s0.z = fmaf(k2.x, v.z, fmaf(-b2.x, q.z, s0.z));
                s0.w = fmaf(k2.x, v.w, fmaf(-b2.x, q.w, s0.w));
                s1.x = fmaf(k2.y, v.x, fmaf(-b2.y, q.x, s1.x));
                s1.y = fmaf(k2.y, v.y, fmaf(-b2.y, q.y, s1.y));
                s1.z = fmaf(k2.y, v.z, fmaf(-b2.y, q.z, s1.z));
                s1.w = fmaf(k2.y, v.w, fmaf(-b2.y, q.w, s1.w));
            }
            *reinterpret_cast<float4*>(Ss + d * DC_EV + cq) = s0;
            *reinterpret_cast<float4*>(Ss + (d + 1) * DC_EV + cq) = s1;
        }
        __syncthreads();                                   // (the stage may be filled again, S is whole)
    }
    pdl_launch_dependents();
    for (int idx = tid; idx < D * DC_EV; idx += blockDim.x) {
        const int d = idx / DC_EV, e = e0 + idx % DC_EV;
        if (e < Dv) gS[(size_t)d * Dv + e] = Ss[idx];
    }
}

static size_t dc_scan_smem(int D, int stages) {
    const size_t Dp = dc_pad(D);
    const size_t stage = (size_t)2 * DC_C * (Dp + 4) + 2 * DC_C * Dp + 3 * DC_C * DC_C + Dp + DC_C * DC_EV;
    return (Dp * DC_EV + DC_C * DC_EV + stages * stage) * sizeof(float);
}

template <typename T>
static int launch_delta_chunk(const DeltaChunkArgs& c, int num_seqs, cudaStream_t st) {
    if (num_seqs <= 0 || c.num_tiles <= 0) return 0;
    const DeltaRuleArgs& a = c.a;
    int rc = dr_check(a);
    if (rc != 0) return rc;
    if (a.out == nullptr || c.work == nullptr || c.tile_seq == nullptr || c.tile_row0 == nullptr ||
        ((uintptr_t)c.work & 15) || ((uintptr_t)a.out & 15) || a.decay_coef > 2.0f)
        return SLB_ERR_BAD_ARG;
    if (num_seqs > 65535) return SLB_ERR_TOO_LARGE;
    const int Dp = dc_pad(a.D), vz = (a.Dv + DC_EV - 1) / DC_EV;
    const size_t smem1 = ((size_t)5 * DC_C * (Dp + 4) + 64 * 68) * sizeof(float);
    static unsigned long long conf1 = 0, conf2 = 0, conf3 = 0;
    rc = slb_configure(&conf1, delta_chunk_prep_kernel<T>, ((size_t)5 * DC_C * (DR_MAX_D + 4) + 64 * 68) * sizeof(float));
    if (rc != 0) return rc;
    rc = slb_launch(delta_chunk_prep_kernel<T>, dim3(c.num_tiles, a.H), dim3(256), smem1, st, c);
    if (rc != 0) return rc;
    if (a.D <= 128) {
        rc = slb_configure(&conf2, delta_chunk_scan_kernel<T, 2>, dc_scan_smem(128, 2));
        if (rc != 0) return rc;
        return slb_launch(delta_chunk_scan_kernel<T, 2>, dim3(num_seqs, a.H, vz), dim3(256), dc_scan_smem(a.D, 2), st, c);
    }
    rc = slb_configure(&conf3, delta_chunk_scan_kernel<T, 1>, dc_scan_smem(DR_MAX_D, 1));
    if (rc != 0) return rc;
    return slb_launch(delta_chunk_scan_kernel<T, 1>, dim3(num_seqs, a.H, vz), dim3(256), dc_scan_smem(a.D, 1), st, c);
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
int slb_delta_chunk_tokens() { return DC_C; }
int slb_delta_chunk_work_floats(int D) { return (int)dc_floats(D); }
int slb_delta_chunk_f32(const DeltaChunkArgs* c, int num_seqs, cudaStream_t st) {
    return launch_delta_chunk<float>(*c, num_seqs, st);
}
int slb_delta_chunk_bf16(const DeltaChunkArgs* c, int num_seqs, cudaStream_t st) {
    return launch_delta_chunk<bf16>(*c, num_seqs, st);
}
}
