// A gated linear recurrence, one number of state a channel (float32, in a state slot):
//
//     log a_t = rate r_t,   S_t = a_t S_{t-1} + sqrt(1 - a_t^2) i_t u_t,   out_t = S_t gelu_tanh(y_t + b_y)
//
// with r_t = sigmoid(z^r_t + b_r), i_t = sigmoid(z^i_t + b_i) and rate = -coef softplus(lambda) <= 0 per
// channel.  u (behind its convolution) and y have the compute type; the gates' logits z are float32 and
// come from block-diagonal products: block b of n channels has its logits at z + b * z_block +
// token * z_token, n for r and then n for i.  Everything here is float32; S is zero for a new request.
//
// Steps of single tokens: a thread a (request, channel).
//
// Token by token (float32 rows): a block owns 16 channels of a request and takes
// its tokens 64 at a time: all threads form a and the update of every (token, channel), 16 threads walk
// the tokens (one multiply-add each, in order, so the result of a token does not depend on how the
// request was cut), all threads finish the outputs.
//
// In segments (bfloat16 rows of longer portions): 32 segments of 8 tokens at a time, a thread a (segment,
// channel).  A segment is S -> A S + B; each thread forms its own pair, takes the segments before it
// from shared memory, and walks its tokens once more from the state that enters.
#include "common.cuh"

#define GR_EC 16
#define GR_TT 64

struct GatedRecArgs {
    const void* u; int ldu;
    const float* z; long long z_block, z_token;
    const float* r_bias; const float* i_bias; const float* rate;
    const void* y; int ldy; const float* y_bias;
    float* state; long long state_stride; int num_slots;
    const int* cu_q; const int* state_slots;
    int width, n;
    void* out; int ldo;
};

__device__ __forceinline__ float gr_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float gr_gelu_tanh(float z) {
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
// a and sqrt(1 - a^2) from log a (1 - a^2 = -expm1(2 log a): no cancellation for a near 1)
__device__ __forceinline__ void gr_decay(float log_a, float& a, float& gain) {
    a = decay_exp(log_a);
    gain = sqrtf(-expm1f(2.0f * log_a));
}

template <typename T>
__global__ void __launch_bounds__(256) gated_recurrence_kernel(const GatedRecArgs g) {
    __shared__ float sa[GR_TT][GR_EC], sb[GR_TT][GR_EC];
    pdl_wait();
    pdl_launch_dependents();
    const int s = blockIdx.x, c0 = blockIdx.y * GR_EC;
    const int q0 = g.cu_q[s];
    const int qlen = g.cu_q[s + 1] - q0;
    if (qlen <= 0) return;
    const int slot = g.state_slots[s];
    if (slot < 0 || slot >= g.num_slots) return;
    const int tid = threadIdx.x, ch = tid % GR_EC, tk = tid / GR_EC;
    const int c = c0 + ch;
    const bool live = c < g.width;
    const T* u = reinterpret_cast<const T*>(g.u);
    const T* y = reinterpret_cast<const T*>(g.y);
    T* out = reinterpret_cast<T*>(g.out);
    float rb = 0.f, ib = 0.f, rate = 0.f, yb = 0.f;
    const float* z = g.z;
    if (live) {
        rb = g.r_bias[c]; ib = g.i_bias[c]; rate = g.rate[c]; yb = g.y_bias[c];
        const int b = c / g.n;
        z += (size_t)b * g.z_block + (c - b * g.n);
    }
    float* sp = g.state + (size_t)slot * g.state_stride + c;
    float S = live && tk == 0 ? *sp : 0.f;
    constexpr int PER = 256 / GR_EC;             // tokens in flight
    for (int t0 = 0; t0 < qlen; t0 += GR_TT) {
        const int n = min(GR_TT, qlen - t0);
#pragma unroll
        for (int i = 0; i < GR_TT / PER; ++i) {
            const int j = tk + i * PER;
            if (j < n && live) {
                const size_t t = q0 + t0 + j;
                const float r = gr_sigmoid(z[t * g.z_token] + rb);
                const float in = gr_sigmoid(z[t * g.z_token + g.n] + ib);
                float a, gain;
                gr_decay(rate * r, a, gain);
                sa[j][ch] = a;
                sb[j][ch] = gain * in * to_float(u[t * g.ldu + c]);
            }
        }
        __syncthreads();
        if (tk == 0 && live) {
#pragma unroll 8
            for (int j = 0; j < n; ++j) {
                S = fmaf(sa[j][ch], S, sb[j][ch]);
                sb[j][ch] = S;
            }
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < GR_TT / PER; ++i) {
            const int j = tk + i * PER;
            if (j < n && live) {
                const size_t t = q0 + t0 + j;
                out[t * g.ldo + c] = from_float<T>(sb[j][ch] * gr_gelu_tanh(to_float(y[t * g.ldy + c]) + yb));
            }
        }
        // (a thread overwrites only the elements of sa and sb that it has just read itself, and the
        // walk over them comes after the next barrier)
    }
    if (tk == 0 && live) *sp = S;
}

template <typename T>
__global__ void __launch_bounds__(128) gated_recurrence_step_kernel(const GatedRecArgs g) {
    pdl_wait();
    pdl_launch_dependents();
    const int s = blockIdx.x, c = blockIdx.y * 128 + threadIdx.x;
    const int q0 = g.cu_q[s], q1 = g.cu_q[s + 1];
    const int slot = g.state_slots[s];
    if (q1 <= q0 || slot < 0 || slot >= g.num_slots || c >= g.width) return;
    const float rb = g.r_bias[c], ib = g.i_bias[c], rate = g.rate[c], yb = g.y_bias[c];
    const int b = c / g.n;
    const float* z = g.z + (size_t)b * g.z_block + (c - b * g.n);
    float* sp = g.state + (size_t)slot * g.state_stride + c;
    float S = *sp;
    for (size_t t = q0; t < q1; ++t) {
        const float r = gr_sigmoid(z[t * g.z_token] + rb);
        const float in = gr_sigmoid(z[t * g.z_token + g.n] + ib);
        float a, gain;
        gr_decay(rate * r, a, gain);
        S = fmaf(a, S, __fmul_rn(__fmul_rn(gain, in), to_float(reinterpret_cast<const T*>(g.u)[t * g.ldu + c])));
        const float y = gr_gelu_tanh(to_float(reinterpret_cast<const T*>(g.y)[t * g.ldy + c]) + yb);
        reinterpret_cast<T*>(g.out)[t * g.ldo + c] = from_float<T>(S * y);
    }
    *sp = S;
}

#define GR_SEGS 32
#define GR_SEG_TOKENS 8

template <typename T>
__global__ void __launch_bounds__(GR_EC * GR_SEGS) gated_recurrence_segments_kernel(const GatedRecArgs g) {
    __shared__ float2 pairs[2][GR_SEGS][GR_EC];
    pdl_wait();
    pdl_launch_dependents();
    const int s = blockIdx.x, c0 = blockIdx.y * GR_EC;
    const int q0 = g.cu_q[s];
    const int qlen = g.cu_q[s + 1] - q0;
    if (qlen <= 0) return;
    const int slot = g.state_slots[s];
    if (slot < 0 || slot >= g.num_slots) return;
    const int ch = threadIdx.x % GR_EC, seg = threadIdx.x / GR_EC;
    const int c = c0 + ch;
    const bool live = c < g.width;
    const T* u = reinterpret_cast<const T*>(g.u);
    const T* y = reinterpret_cast<const T*>(g.y);
    T* out = reinterpret_cast<T*>(g.out);
    float rb = 0.f, ib = 0.f, rate = 0.f, yb = 0.f, S = 0.f;
    const float* z = g.z;
    float* sp = g.state + (size_t)slot * g.state_stride + c;
    if (live) {
        rb = g.r_bias[c]; ib = g.i_bias[c]; rate = g.rate[c]; yb = g.y_bias[c];
        const int b = c / g.n;
        z += (size_t)b * g.z_block + (c - b * g.n);
        S = *sp;
    }
    for (int t0 = 0, k = 0; t0 < qlen; t0 += GR_SEGS * GR_SEG_TOKENS, ++k) {
        const int first = t0 + seg * GR_SEG_TOKENS;
        float zr[GR_SEG_TOKENS], zi[GR_SEG_TOKENS], uv[GR_SEG_TOKENS], yv[GR_SEG_TOKENS];
#pragma unroll
        for (int i = 0; i < GR_SEG_TOKENS; ++i) {
            zr[i] = zi[i] = uv[i] = yv[i] = 0.f;
            if (live && first + i < qlen) {
                const size_t t = q0 + first + i;
                zr[i] = z[t * g.z_token];
                zi[i] = z[t * g.z_token + g.n];
                uv[i] = to_float(u[t * g.ldu + c]);
                yv[i] = to_float(y[t * g.ldy + c]);
            }
        }
        float A = 1.f, B = 0.f;                  // (zr becomes a, zi the update)
#pragma unroll
        for (int i = 0; i < GR_SEG_TOKENS; ++i) {
            float a = 1.f, b = 0.f;
            if (live && first + i < qlen) {
                float gain;
                gr_decay(rate * gr_sigmoid(zr[i] + rb), a, gain);
                b = gain * gr_sigmoid(zi[i] + ib) * uv[i];
            }
            zr[i] = a;
            zi[i] = b;
            A *= a;
            B = fmaf(a, B, b);
        }
        float2 (*row)[GR_EC] = pairs[k & 1];     // (two buffers: one barrier a round)
        row[seg][ch] = make_float2(A, B);
        __syncthreads();
        float enter = S;
#pragma unroll 8
        for (int i = 0; i < GR_SEGS; ++i) {
            if (i == seg) enter = S;
            const float2 p = row[i][ch];
            S = fmaf(p.x, S, p.y);
        }
#pragma unroll
        for (int i = 0; i < GR_SEG_TOKENS; ++i) {
            enter = fmaf(zr[i], enter, zi[i]);
            if (live && first + i < qlen)
                out[(size_t)(q0 + first + i) * g.ldo + c] = from_float<T>(enter * gr_gelu_tanh(yv[i] + yb));
        }
    }
    if (seg == 0 && live) *sp = S;
}

template <typename T>
static int launch_gated_recurrence(const GatedRecArgs& g, int num_seqs, int form, cudaStream_t st) {
    if (num_seqs <= 0) return 0;
    if (g.width <= 0 || g.n <= 0 || g.width % g.n || g.u == nullptr || g.z == nullptr || g.y == nullptr ||
        g.state == nullptr || g.state_stride < g.width || g.num_slots <= 0 || g.r_bias == nullptr ||
        g.i_bias == nullptr || g.rate == nullptr || g.y_bias == nullptr || g.out == nullptr)
        return SLB_ERR_BAD_ARG;
    const int gy = (g.width + GR_EC - 1) / GR_EC;
    if (gy > 65535) return SLB_ERR_TOO_LARGE;
    if (form == 2)
        return slb_launch(gated_recurrence_step_kernel<T>, dim3(num_seqs, (g.width + 127) / 128), dim3(128), 0, st, g);
    if (form == 1)
        return slb_launch(gated_recurrence_segments_kernel<T>, dim3(num_seqs, gy), dim3(GR_EC * GR_SEGS), 0, st, g);
    return slb_launch(gated_recurrence_kernel<T>, dim3(num_seqs, gy), dim3(256), 0, st, g);
}

extern "C" {
// form 0: token by token, 1: in segments, 2: single tokens
int slb_gated_recurrence_f32(const GatedRecArgs* g, int num_seqs, int form, cudaStream_t st) {
    return launch_gated_recurrence<float>(*g, num_seqs, form, st);
}
int slb_gated_recurrence_bf16(const GatedRecArgs* g, int num_seqs, int form, cudaStream_t st) {
    return launch_gated_recurrence<bf16>(*g, num_seqs, form, st);
}
}
