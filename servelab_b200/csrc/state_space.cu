// Selective state space (the recurrence of Mamba-2) over a per-request state, token by token:
//
//     dt = softplus(z_t + dt_bias_h)
//     S_t = exp(-rate_h dt) S_{t-1} + dt B_t x_t^T        (S: N x P a head, float32, kept in a state slot)
//     y_t = S_t^T C_t + skip_h x_t
//
// with B and C shared by the heads of a group.  Everything after the load is float32.
//
// A block owns (request, head, a slice of the value columns).  Its threads form a grid of `RT` row threads by
// 256 / RT column threads of V neighbouring columns each; a row thread keeps the state elements of the rows
// n = i * RT + row in registers, so a warp's accesses to the state are whole lines.  Tokens are taken in order,
// SS_TT at a time, their B, C and x rows staged in shared memory; the row threads' parts of an output are
// added in a fixed order.  The state is read at the start and written at the end: a request may be cut
// anywhere, and a token's result is bit-identical however the prompt is cut and whatever else is in the
// batch.  A step of single tokens is one read and one write of the state.
#include "state_space.cuh"

#define SS_THREADS 256
#define SS_TT 8
#define SS_MAX_N 256

template <typename T, int V, int RT, int R>
__global__ void __launch_bounds__(SS_THREADS) state_space_kernel(const StateSpaceArgs a) {
    constexpr int CT = SS_THREADS / RT, EC = CT * V;       // column threads, columns a block
    extern __shared__ float ss_smem[];
    pdl_wait();
    pdl_launch_dependents();
    const int s = blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * EC;
    const int q0 = a.cu_q[s];
    const int qlen = a.cu_q[s + 1] - q0;
    if (qlen <= 0) return;
    const int slot = a.state_slots[s];
    if (slot < 0 || slot >= a.num_slots) return;
    const int N = a.N, P = a.P, grp = h / (a.H / a.G);
    const int tid = threadIdx.x, ct = tid % CT, rt = tid / CT;
    const int col = e0 + ct * V;
    const bool live = col < P;                             // (V > 1: P is a multiple of V)
    float* srow = a.state + (size_t)slot * (size_t)a.state_stride + (size_t)h * N * P;

    float* bs = ss_smem;                                   // [SS_TT][N]
    float* cs = bs + SS_TT * N;                            // [SS_TT][N]
    float* xs = cs + SS_TT * N;                            // [SS_TT][EC]
    float* part = xs + SS_TT * EC;                         // [SS_TT][RT][EC]
    float* dts = part + SS_TT * RT * EC;                   // [SS_TT] step sizes, then [SS_TT] decays
    float* dec = dts + SS_TT;

    float st[R][V];
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int n = i * RT + rt;
        const bool ok = live && n < N;
        if constexpr (V == 4) {
            const float4 v = ok ? *reinterpret_cast<const float4*>(srow + (size_t)n * P + col) : make_float4(0.f, 0.f, 0.f, 0.f);
            st[i][0] = v.x; st[i][1] = v.y; st[i][2] = v.z; st[i][3] = v.w;
        } else {
            st[i][0] = ok ? srow[(size_t)n * P + col] : 0.f;
        }
    }
    const T* u = reinterpret_cast<const T*>(a.u);
    const float skip = a.skip[h], rate = a.rate[h], dt_bias = a.dt_bias[h];
    for (int t0 = 0; t0 < qlen; t0 += SS_TT) {
        const int n_tok = min(SS_TT, qlen - t0);
        for (int idx = tid; idx < n_tok * N; idx += SS_THREADS) {
            const int j = idx / N, n = idx - j * N;
            const T* row = u + (size_t)(q0 + t0 + j) * a.ld + grp * N + n;
            bs[idx] = to_float(row[a.b_off]);
            cs[idx] = to_float(row[a.c_off]);
        }
        for (int idx = tid; idx < n_tok * EC; idx += SS_THREADS) {
            const int j = idx / EC, c = e0 + (idx - j * EC);
            xs[idx] = c < P ? to_float(u[(size_t)(q0 + t0 + j) * a.ld + a.x_off + (size_t)h * P + c]) : 0.f;
        }
        if (tid < n_tok) {
            const float d = ss_step(a.dt[(size_t)(q0 + t0 + tid) * a.ld_dt + h] + dt_bias);
            dts[tid] = d;
            dec[tid] = decay_exp(-rate * d);
        }
        __syncthreads();
        for (int j = 0; j < n_tok; ++j) {
            const float d = dts[j], g = dec[j];
            float xd[V], acc[V];
#pragma unroll
            for (int v = 0; v < V; ++v) {
                xd[v] = d * xs[j * EC + ct * V + v];
                acc[v] = 0.f;
            }
#pragma unroll
            for (int i = 0; i < R; ++i) {
                const int n = i * RT + rt;
                if (n < N) {
                    const float b = bs[j * N + n], c = cs[j * N + n];
#pragma unroll
                    for (int v = 0; v < V; ++v) {
                        st[i][v] = fmaf(g, st[i][v], b * xd[v]);
                        acc[v] = fmaf(st[i][v], c, acc[v]);
                    }
                }
            }
#pragma unroll
            for (int v = 0; v < V; ++v) part[(j * RT + rt) * EC + ct * V + v] = acc[v];
        }
        __syncthreads();
        for (int idx = tid; idx < n_tok * EC; idx += SS_THREADS) {
            const int j = idx / EC, c = idx - j * EC;
            if (e0 + c < P) {
                float y = skip * xs[idx];
#pragma unroll
                for (int r = 0; r < RT; ++r) y += part[(j * RT + r) * EC + c];
                a.out[(size_t)(q0 + t0 + j) * a.ldo + (size_t)h * P + e0 + c] = y;
            }
        }
        __syncthreads();                                   // (xs and part are written again)
    }
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int n = i * RT + rt;
        if (live && n < N) {
            if constexpr (V == 4)
                *reinterpret_cast<float4*>(srow + (size_t)n * P + col) = make_float4(st[i][0], st[i][1], st[i][2], st[i][3]);
            else
                srow[(size_t)n * P + col] = st[i][0];
        }
    }
}

template <typename T, int V, int RT, int R>
static int launch_state_space_form(const StateSpaceArgs& a, int num_seqs, cudaStream_t st) {
    constexpr int EC = SS_THREADS / RT * V;
    const size_t smem = ((size_t)2 * SS_TT * a.N + SS_TT * EC + SS_TT * RT * EC + 2 * SS_TT) * sizeof(float);
    const size_t smem_max = ((size_t)2 * SS_TT * SS_MAX_N + SS_TT * EC + SS_TT * RT * EC + 2 * SS_TT) * sizeof(float);
    static unsigned long long configured = 0;
    const int rc = slb_configure(&configured, state_space_kernel<T, V, RT, R>, smem_max);
    if (rc != 0) return rc;
    return slb_launch(state_space_kernel<T, V, RT, R>, dim3(num_seqs, a.H, (a.P + EC - 1) / EC), dim3(SS_THREADS), smem,
                      st, a);
}

template <typename T>
static int launch_state_space(const StateSpaceArgs* in, int num_seqs, cudaStream_t st) {
    if (num_seqs <= 0) return 0;
    const StateSpaceArgs& a = *in;
    if (a.H <= 0 || a.P <= 0 || a.N <= 0 || a.G <= 0 || a.H % a.G != 0 || a.num_slots <= 0 ||
        a.state_stride < (long long)a.H * a.N * a.P || a.ldo < a.H * a.P || a.ld_dt < a.H)
        return SLB_ERR_BAD_ARG;
    if (a.N > SS_MAX_N || a.H > 65535 || a.P > 65535) return SLB_ERR_TOO_LARGE;
    if (a.P % 4 == 0 && a.state_stride % 4 == 0 && ((uintptr_t)a.state & 15) == 0) {
        if (a.N <= 64) return launch_state_space_form<T, 4, 16, 4>(a, num_seqs, st);
        if (a.N <= 128) return launch_state_space_form<T, 4, 16, 8>(a, num_seqs, st);
        return launch_state_space_form<T, 4, 16, 16>(a, num_seqs, st);
    }
    if (a.N <= 64) return launch_state_space_form<T, 1, 8, 8>(a, num_seqs, st);
    return launch_state_space_form<T, 1, 8, 32>(a, num_seqs, st);
}

extern "C" {
int slb_state_space_max_state() { return SS_MAX_N; }
int slb_state_space_f32(const StateSpaceArgs* a, int num_seqs, cudaStream_t st) {
    return launch_state_space<float>(a, num_seqs, st);
}
int slb_state_space_bf16(const StateSpaceArgs* a, int num_seqs, cudaStream_t st) {
    return launch_state_space<bf16>(a, num_seqs, st);
}
}
