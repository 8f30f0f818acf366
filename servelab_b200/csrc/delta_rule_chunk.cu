// The delta rule of delta_rule.cu over longer portions, in chunks of C = 32 tokens.
//
// With the entering state S, L_t the sum of log w up to and including token t (per channel),
// G_t = e^(L_t), seen_t = u_t^T S_{t-1} and b_t = a_t u_t,
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
// r_t G_t, k_j G_C / G_j, b_j G_C / G_j and G_C in a work buffer, padded as the second launch wants them
// in shared memory; `scan` walks a request's chunks with 16 value columns of the state a block, a
// chunk's record fetched as one bulk copy while the one before is worked on.
//
// The products run on mma.sync with every float32 operand split into two TF32 numbers (the
// product of the two low parts is left out: it is below float32's own rounding);
// bfloat16 values need one); everything else, the solve and the decays included, is float32.
#include "delta_rule.cuh"
#include "mma_util.cuh"

#define DC_C 32
#define DC_EV 16
#define DC_LM 36                             // row stride of Y, P, Q and of the [value][token] operands

struct DeltaChunkArgs {
    DeltaRuleArgs a;
    const int* tile_seq; const int* tile_row0; int num_tiles;
    float* work;                             // [num_tiles][H][dc_floats(D)]
};

// A (chunk, head)'s record: X, R [C][Dp + 4], K, B [C][Dp + 8], Y, P, Q [C][36], G_C [Dp].  The strides
// put the 32 lanes of an operand fragment on 32 banks: 4 g + t where the contraction runs along a row,
// 8 t + g where it runs down the rows.
__host__ __device__ constexpr int dc_pad(int D) { return (D + 15) & ~15; }
__host__ __device__ constexpr int dc_lx(int D) { return dc_pad(D) + 4; }
__host__ __device__ constexpr int dc_lk(int D) { return dc_pad(D) + 8; }
__host__ __device__ constexpr int dc_floats(int D) {
    return DC_C * (2 * dc_lx(D) + 2 * dc_lk(D) + 3 * DC_LM) + dc_pad(D);
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
    const int D = a.D, Dp = dc_pad(D), LX = dc_lx(D), LK = dc_lk(D);
    float* Ls = dc_smem;                         // [C][LX]: log decays, then their running sums
    float* Rs = Ls + DC_C * LX;                  // r_t G_t          (rows 0..31 of the left operand)
    float* Us = Rs + DC_C * LX;                  // u_t G_{t-1}      (rows 32..63)
    float* Ks = Us + DC_C * LX;                  // k_j / G_j        (rows 0..31 of the right operand)
    float* Bs = Ks + DC_C * LX;                  // a_j u_j / G_j    (rows 32..63)
    float* Gm = Bs + DC_C * LX;                  // [32][68]: N | M
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    {
        const T* row = reinterpret_cast<const T*>(a.proj) + (size_t)t0 * a.ld + h * D;
        const float* zrow = a.gate_z + (size_t)t0 * a.ld_gate + h * D;
for (int d = lane; d < Dp; d += 32) {        // (a warp has the four rows from 4 warp)
            const bool live = d < D;
            const float ab = live ? a.a_bias[h * D + d] : 0.f;
            float l[4], k[4], r[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int j = warp * 4 + i;
                l[i] = k[i] = r[i] = b[i] = 0.f;
                if (live && j < n) {
                    const T* p = row + (size_t)j * a.ld + d;
                    l[i] = zrow[(size_t)j * a.ld_gate + d];
                    k[i] = to_float(p[a.k_off]);
                    r[i] = to_float(p[a.r_off]);
                    b[i] = to_float(p[a.a_off]);
                }
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int at = (warp * 4 + i) * LX + d;
                const bool in = live && warp * 4 + i < n;
                Ls[at] = in ? -a.decay_coef * dr_sigmoid(l[i]) : 0.f;
                Ks[at] = k[i];
                Rs[at] = r[i];
                Bs[at] = in ? dr_sigmoid(b[i] + ab) : 0.f;
            }
        }
    }
    __syncthreads();
    for (int d = tid; d < Dp; d += 256) {
        float l[DC_C], run = 0.f;
#pragma unroll
        for (int j = 0; j < DC_C; ++j) l[j] = Ls[j * LX + d];
#pragma unroll
        for (int j = 0; j < DC_C; ++j) Ls[j * LX + d] = run += l[j];    // (beyond the tokens the sum stays what it is)
    }
    __syncthreads();
    float* rec = c.work + ((size_t)tile * a.H + h) * dc_floats(D);
    float* gX = rec, *gR = gX + DC_C * LX, *gK = gR + DC_C * LX, *gB = gK + DC_C * LK;
    float* gY = gB + DC_C * LK, *gP = gY + DC_C * DC_LM, *gQ = gP + DC_C * DC_LM, *gG = gQ + DC_C * DC_LM;
    {
        const int j0 = warp * 4;
        float inv[4] = {};
        for (int d = lane; d < Dp; d += 32)
#pragma unroll
            for (int i = 0; i < 4; ++i) inv[i] = fmaf(Ks[(j0 + i) * LX + d], Ks[(j0 + i) * LX + d], inv[i]);
#pragma unroll
        for (int i = 0; i < 4; ++i) inv[i] = 1.0f / sqrtf(warp_sum(inv[i]) + a.unit_eps);
        for (int d = lane; d < Dp; d += 32) {
            const float Le = Ls[(DC_C - 1) * LX + d];
            float before = j0 > 0 ? expf(Ls[(j0 - 1) * LX + d]) : 1.0f;
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int at = (j0 + i) * LX + d;
                const float L = Ls[at], k = Ks[at], u = k * inv[i], b = Bs[at] * u;
                const float now = expf(L), up = expf(-L), rest = expf(Le - L), rg = Rs[at] * now;
                Rs[at] = rg;
                Us[at] = u * before;
                Ks[at] = k * up;
                Bs[at] = b * up;
                gR[at] = rg;
                gK[(j0 + i) * LK + d] = k * rest;
                gB[(j0 + i) * LK + d] = b * rest;
                before = now;
            }
        }
    }
    for (int d = tid; d < Dp; d += 256) gG[d] = decay_exp(Ls[(DC_C - 1) * LX + d]);
    __syncthreads();
    // [R; U] [K; B]^T, 64 x 64: a warp has 16 rows and 32 columns
    {
        const int g = lane >> 2, t = lane & 3, m0 = (warp >> 1) * 16, n0 = (warp & 1) * 32;
        float acc[4][4] = {}, low[4][4] = {};
        const float* A = Rs + (m0 + g) * LX + t;     // (Us follows Rs, Bs follows Ks)
        const float* B = Ks + (n0 + g) * LX + t;
#pragma unroll 2
        for (int d = 0; d < Dp; d += 8) {
            unsigned ah[4], al[4];
#pragma unroll
            for (int i = 0; i < 4; ++i)
                slb_mma::split_tf32(A[(i & 1) * 8 * LX + d + (i >> 1) * 4], ah[i], al[i]);
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                unsigned bh[2], bl[2];
                slb_mma::split_tf32(B[q * 8 * LX + d], bh[0], bl[0]);
                slb_mma::split_tf32(B[q * 8 * LX + d + 4], bh[1], bl[1]);
                slb_mma::mma_tf32(low[q], al, bh);
                slb_mma::mma_tf32(acc[q], ah, bh);
                slb_mma::mma_tf32(low[q], ah, bl);
            }
        }
#pragma unroll
        for (int q = 0; q < 4; ++q)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int r = m0 + g + (i >> 1) * 8, jj = q * 8 + 2 * t + (i & 1), tt = r & 31;
                const float v = acc[q][i] + low[q][i];
                if (r < 32) (n0 == 0 ? gP : gQ)[tt * DC_LM + jj] = jj <= tt ? v : 0.f;
                else Gm[tt * 68 + n0 + jj] = jj < tt ? v : 0.f;
            }
    }
    __syncthreads();
    // (I + M) z = rhs, a column a thread: the Dp columns of u G_{t-1} give X, the 32 of N give Y
    for (int col = tid; col < Dp + DC_C; col += 256) {
        float z[DC_C];
        const bool isX = col < Dp;
#pragma unroll
        for (int t = 0; t < DC_C; ++t) {
            float v = isX ? Us[t * LX + col] : Gm[t * 68 + (col - Dp)];
            const float* m = Gm + t * 68 + 32;
#pragma unroll
            for (int j4 = 0; j4 < (t + 3) / 4; ++j4) {     // (M is zero from column t on)
                const float4 m4 = *reinterpret_cast<const float4*>(m + 4 * j4);
                v = fmaf(-m4.x, z[4 * j4], v);
                if (4 * j4 + 1 < t) v = fmaf(-m4.y, z[4 * j4 + 1], v);
                if (4 * j4 + 2 < t) v = fmaf(-m4.z, z[4 * j4 + 2], v);
                if (4 * j4 + 3 < t) v = fmaf(-m4.w, z[4 * j4 + 3], v);
            }
            z[t] = v;
            if (isX) gX[t * LX + col] = v;
            else gY[t * DC_LM + col - Dp] = v;
        }
    }
}

// acc += A B over `steps` contraction steps of 8, the cross terms of the split in chains of their own
// (low).  A's fragment starts at A (+ row8 for the row 8 below, + k4 for the contraction 4 further, + k8 a
// step); B is [column][contraction] with stride ldb, B already at this lane's column and contraction, NT
// tiles of 8 columns; EXACT: B's elements are TF32 numbers.
template <int NT, bool EXACT>
__device__ __forceinline__ void dc_product(float (&acc)[NT][4], float (&low)[2][NT][4], const float* A, int row8,
                                           int k4, int k8, const float* B, int ldb, int steps) {
#pragma unroll 8
    for (int s = 0; s < steps; ++s) {
        unsigned ah[4], al[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) slb_mma::split_tf32(A[s * k8 + (i & 1) * row8 + (i >> 1) * k4], ah[i], al[i]);
#pragma unroll
        for (int q = 0; q < NT; ++q) {
            unsigned bh[2], bl[2];
            slb_mma::split_tf32(B[q * 8 * ldb + s * 8], bh[0], bl[0]);
            slb_mma::split_tf32(B[q * 8 * ldb + s * 8 + 4], bh[1], bl[1]);
            slb_mma::mma_tf32(low[0][q], al, bh);
            slb_mma::mma_tf32(acc[q], ah, bh);
            if (!EXACT) slb_mma::mma_tf32(low[1][q], ah, bl);
        }
    }
}

// S <- G S + K^T V + B^T (-seen) for the 16 rows from d0 and NT tiles of 8 value columns from n0
template <int NT, bool EXACT>
__device__ __forceinline__ void dc_update(float* Ss, int LX, const float* G, const float* Kd, const float* Bd, int LK,
                                          const float* Vt, const float* Nt, int d0, int n0, int g, int t) {
    float acc[NT][4] = {}, low[2][NT][4] = {};
    dc_product<NT, EXACT>(acc, low, Kd + t * LK + d0 + g, 8, 4 * LK, 8 * LK, Vt + (n0 + g) * DC_LM + t, DC_LM, DC_C / 8);
    dc_product<NT, false>(acc, low, Bd + t * LK + d0 + g, 8, 4 * LK, 8 * LK, Nt + (n0 + g) * DC_LM + t, DC_LM, DC_C / 8);
    const float g0 = G[d0 + g], g1 = G[d0 + g + 8];
#pragma unroll
    for (int q = 0; q < NT; ++q)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            float* s = Ss + (n0 + q * 8 + 2 * t + (i & 1)) * LX + d0 + g + (i >> 1) * 8;
            *s = fmaf(i >> 1 ? g1 : g0, *s, acc[q][i] + (low[0][q][i] + low[1][q][i]));
        }
}

// STAGES 2: the next chunk's record is fetched while this one is worked on.
template <typename T, int STAGES>
__global__ void __launch_bounds__(256) delta_chunk_scan_kernel(const DeltaChunkArgs c) {
    extern __shared__ __align__(16) float dc_smem[];
    constexpr bool EXACT = sizeof(T) == 2;           // (a bfloat16 value is a TF32 number)
    __shared__ int first_s;
    __shared__ __align__(8) uint64_t bars[STAGES];
    pdl_wait();
    const DeltaRuleArgs& a = c.a;
    const int s = blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * DC_EV;
    const int q0 = a.cu_q[s];
    const int qlen = a.cu_q[s + 1] - q0;
    if (qlen <= 0) return;
    const int slot = a.state_slots[s];
    if (slot < 0 || slot >= a.num_slots) return;
    const int tid = threadIdx.x;
    if (tid == 0) {
        first_s = c.num_tiles;
        for (int i = 0; i < STAGES; ++i) slb_mma::mbar_init(&bars[i], 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    for (int i = tid; i < c.num_tiles; i += 256)     // a request's chunks are neighbours in the list, in order
        if (c.tile_seq[i] == s) { atomicMin(&first_s, i); break; }
    __syncthreads();
    const int first = first_s;
    const int count = (qlen + DC_C - 1) / DC_C;
    if (first + count > c.num_tiles) return;
    const int D = a.D, Dv = a.Dv, Dp = dc_pad(D), LX = dc_lx(D), LK = dc_lk(D);
    const int rec_floats = dc_floats(D);
    float* stages = dc_smem;
    float* Ss = stages + STAGES * rec_floats;        // [EV][LX]: the state's columns
    float* Nt = Ss + DC_EV * LX;                     // [EV][LM]: -seen
    float* Vts = Nt + DC_EV * DC_LM;                 // [2][EV][LM]
    const float* recs = c.work + ((size_t)first * a.H + h) * rec_floats;
    auto fetch = [&](int k) {
        slb_mma::mbar_arrive_expect_tx(&bars[k % STAGES], (uint32_t)rec_floats * 4);
        slb_mma::bulk_copy_g2s(stages + (k % STAGES) * rec_floats, recs + (size_t)k * a.H * rec_floats,
                               (uint32_t)rec_floats * 4, &bars[k % STAGES]);
    };
    if (tid == 0) fetch(0);
    float* gS = a.state + (size_t)slot * a.state_stride + (size_t)h * D * Dv;
    for (int idx = tid; idx < Dp * DC_EV; idx += 256) {
        const int d = idx / DC_EV, e = idx % DC_EV;
        Ss[e * LX + d] = d < D && e0 + e < Dv ? gS[(size_t)d * Dv + e0 + e] : 0.f;
    }
    // the values of a chunk: two (token, column) pairs a thread, kept in registers on their way
    const T* vp = reinterpret_cast<const T*>(a.proj) + (size_t)q0 * a.ld + a.v_off + h * Dv + e0;
    const int ve = tid % DC_EV, vj = tid / DC_EV;
    float v0, v1;
    auto load_v = [&](int k) {
        const int t = k * DC_C + vj;
        const bool live = e0 + ve < Dv;
        v0 = live && t < qlen ? to_float(vp[(size_t)t * a.ld + ve]) : 0.f;
        v1 = live && t + 16 < qlen ? to_float(vp[(size_t)(t + 16) * a.ld + ve]) : 0.f;
    };
    auto store_v = [&](int k) {
        float* Vt = Vts + (k & 1) * DC_EV * DC_LM + ve * DC_LM + vj;
        Vt[0] = v0;
        Vt[16] = v1;
    };
    load_v(0);
    store_v(0);
    const int warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int m0 = (warp >> 1) * 16, n0 = (warp & 1) * 8;
    for (int k = 0; k < count; ++k) {
        const bool there = slb_mma::mbar_wait(&bars[k % STAGES], (k / STAGES) & 1);
        if (!__syncthreads_and(there)) return;       // (the copy never came: nothing of ours is in flight but it)
        const bool more = k + 1 < count;
        if (STAGES == 2 && more && tid == 0) fetch(k + 1);
        if (more) load_v(k + 1);
        const float* b = stages + (k % STAGES) * rec_floats;
        const float* Kd = b + 2 * DC_C * LX, *Bd = Kd + DC_C * LK, *Ym = Bd + DC_C * LK, *Qm = Ym + 2 * DC_C * DC_LM;
        const float* G = Qm + DC_C * DC_LM, *Vt = Vts + (k & 1) * DC_EV * DC_LM;
        // rows 0..31: X S + Y V = seen; rows 32..63: R S + P V, the outputs without what was removed
        float acc[1][4] = {}, low[2][1][4] = {};
        dc_product<1, false>(acc, low, b + (m0 + g) * LX + t, 8 * LX, 4, 8, Ss + (n0 + g) * LX + t, LX, Dp / 8);
        dc_product<1, EXACT>(acc, low, Ym + (m0 + g) * DC_LM + t, 8 * DC_LM, 4, 8, Vt + (n0 + g) * DC_LM + t, DC_LM,
                             DC_C / 8);
        if (m0 < DC_C) {
#pragma unroll
            for (int i = 0; i < 4; ++i)
                Nt[(n0 + 2 * t + (i & 1)) * DC_LM + m0 + g + (i >> 1) * 8] = -(acc[0][i] + (low[0][0][i] + low[1][0][i]));
        }
        __syncthreads();
        if (m0 >= DC_C) {
            dc_product<1, false>(acc, low, Qm + (m0 - DC_C + g) * DC_LM + t, 8 * DC_LM, 4, 8, Nt + (n0 + g) * DC_LM + t,
                                 DC_LM, DC_C / 8);
            const int e = e0 + n0 + 2 * t;
#pragma unroll
            for (int i = 0; i < 4; i += 2) {
                const int tt = k * DC_C + m0 - DC_C + g + i * 4;
                if (tt >= qlen || e >= Dv) continue;
                float* o = a.out + (size_t)(q0 + tt) * a.ldo + h * Dv + e;
                const float x = acc[0][i] + (low[0][0][i] + low[1][0][i]);
                const float y = acc[0][i + 1] + (low[0][0][i + 1] + low[1][0][i + 1]);
                if ((Dv & 1) == 0 && (a.ldo & 1) == 0) {
                    *reinterpret_cast<float2*>(o) = make_float2(x, y);
                } else {
                    o[0] = x;
                    if (e + 1 < Dv) o[1] = y;
                }
            }
        }
        if (Dp > 64) {
            for (int d0 = warp * 16; d0 < Dp; d0 += 128) dc_update<2, EXACT>(Ss, LX, G, Kd, Bd, LK, Vt, Nt, d0, 0, g, t);
        } else if (m0 < Dp) {
            dc_update<1, EXACT>(Ss, LX, G, Kd, Bd, LK, Vt, Nt, m0, n0, g, t);
        }
        if (more) store_v(k + 1);
        if (STAGES == 1 && more) {
            __syncthreads();
            if (tid == 0) fetch(k + 1);
        }
    }
    __syncthreads();
    pdl_launch_dependents();
    for (int idx = tid; idx < D * DC_EV; idx += 256) {
        const int d = idx / DC_EV, e = idx % DC_EV;
        if (e0 + e < Dv) gS[(size_t)d * Dv + e0 + e] = Ss[e * LX + d];
    }
}

static size_t dc_prep_smem(int D) { return ((size_t)5 * DC_C * dc_lx(D) + DC_C * 68) * sizeof(float); }
static size_t dc_scan_smem(int D, int stages) {
    return ((size_t)stages * dc_floats(D) + DC_EV * dc_lx(D) + 3 * DC_EV * DC_LM) * sizeof(float);
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
    const int vz = (a.Dv + DC_EV - 1) / DC_EV;
    if (num_seqs > 65535 || vz > 65535) return SLB_ERR_TOO_LARGE;
    static unsigned long long conf1 = 0, conf2 = 0, conf3 = 0;
    rc = slb_configure(&conf1, delta_chunk_prep_kernel<T>, dc_prep_smem(DR_MAX_D));
    if (rc != 0) return rc;
    rc = slb_launch(delta_chunk_prep_kernel<T>, dim3(c.num_tiles, a.H), dim3(256), dc_prep_smem(a.D), st, c);
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
int slb_delta_chunk_tokens() { return DC_C; }
int slb_delta_chunk_work_floats(int D) { return dc_floats(D); }
int slb_delta_chunk_f32(const DeltaChunkArgs* c, int num_seqs, cudaStream_t st) {
    return launch_delta_chunk<float>(*c, num_seqs, st);
}
int slb_delta_chunk_bf16(const DeltaChunkArgs* c, int num_seqs, cudaStream_t st) {
    return launch_delta_chunk<bf16>(*c, num_seqs, st);
}
}
