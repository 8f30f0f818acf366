// Kernels that look at a token and the one before it.
//
//   embed_bigram   x = table[id] + pairs[(previous id * mul_prev + id * mul_cur) mod buckets]; a
//                  sequence's first token takes row `buckets` of the second table.  Float32 stream,
//                  and optionally a copy of it in the table's type (the operand of a later product).
//   token_mix      for n learned vectors mu_i: out_i = h + (h_previous - h) * mu_i; h_previous of a
//                  sequence's first token is zero.
//
// The previous token of a portion's first token comes from the request's state record (the id plus
// one as an integer, 0 for none; a row of h as floats), and the block or thread that reads it there
// also leaves the portion's last token in it, so one launch suffices and nobody else touches the
// element.  Tokens that belong to no request (the padding of a captured step) leave every record
// alone.
#include "common.cuh"

// VEC (1 or 4) consecutive elements as floats, in one access
template <typename T, int VEC>
__device__ __forceinline__ void tm_load(const T* p, float (&v)[VEC]) {
    if constexpr (VEC == 1) {
        v[0] = to_float(p[0]);
    } else if constexpr (sizeof(T) == 2) {
        const uint2 u = *reinterpret_cast<const uint2*>(p);
        const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
        const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
        v[0] = lo.x; v[1] = lo.y; v[2] = hi.x; v[3] = hi.y;
    } else {
        const float4 u = *reinterpret_cast<const float4*>(p);
        v[0] = u.x; v[1] = u.y; v[2] = u.z; v[3] = u.w;
    }
}
template <typename T, int VEC>
__device__ __forceinline__ void tm_store(T* p, const float (&v)[VEC]) {
    if constexpr (VEC == 1) {
        p[0] = from_float<T>(v[0]);
    } else if constexpr (sizeof(T) == 2) {
        __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<unsigned*>(&lo), *reinterpret_cast<unsigned*>(&hi));
    } else {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    }
}

template <typename T, int VEC>
__global__ void __launch_bounds__(256) embed_bigram_kernel(
    const int* __restrict__ ids, const int* __restrict__ cu_q, const int* __restrict__ seq_of_token,
    const int* __restrict__ state_slots, int* __restrict__ state, long long state_stride, int num_slots,
    const T* __restrict__ table, int vocab, const T* __restrict__ pairs, long long buckets, long long mul_prev,
    long long mul_cur, float* __restrict__ out, T* __restrict__ copy, int ldc, int h) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    const int s = seq_of_token[t];
    const int first = cu_q[s], end = cu_q[s + 1];
    const int id = ids[t];
    const bool ok = id >= 0 && id < vocab;
    long long prev = -1;
    if (t > first) {
        prev = ids[t - 1];
    } else if (t < end) {
        const int slot = state_slots[s];
        if (slot >= 0 && slot < num_slots) {
            int* sp = state + (size_t)slot * state_stride;
            prev = (long long)*sp - 1;
            __syncthreads();                           // (every thread has read it)
            if (threadIdx.x == 0) *sp = ids[end - 1] + 1;
        }
    }
    long long pr = prev < 0 ? buckets : (prev * mul_prev + (long long)id * mul_cur) % buckets;
    if (pr < 0) pr += buckets;
    const T* row = table + (size_t)(ok ? id : 0) * h;
    const T* prow = pairs + (size_t)pr * h;
    for (int c = threadIdx.x * VEC; c < h; c += blockDim.x * VEC) {
        float x[VEC], y[VEC];
        tm_load<T, VEC>(row + c, x);
        tm_load<T, VEC>(prow + c, y);
#pragma unroll
        for (int i = 0; i < VEC; ++i) x[i] = ok ? x[i] + y[i] : 0.f;
        tm_store<float, VEC>(out + (size_t)t * h + c, x);
        if (copy != nullptr) tm_store<T, VEC>(copy + (size_t)t * ldc + c, x);
    }
}

// out [n][T][w] with n <= TM_MAX mixes; VEC neighbouring columns a thread.
#define TM_MAX 8
template <typename T, int VEC>
__global__ void __launch_bounds__(256) token_mix_kernel(
    const T* __restrict__ x, int ldx, const float* __restrict__ mu, int n, float* __restrict__ prev,
    long long prev_stride, int num_slots, const int* __restrict__ cu_q, const int* __restrict__ seq_of_token,
    const int* __restrict__ state_slots, T* __restrict__ out, int w, int tokens) {
    const int c0 = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
    pdl_launch_dependents();
    pdl_wait();
    if (c0 >= w) return;
    const int t = blockIdx.y;
    const int s = seq_of_token[t];
    const int first = cu_q[s], end = cu_q[s + 1];
    float h[VEC], hp[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
        h[i] = to_float(x[(size_t)t * ldx + c0 + i]);
        hp[i] = 0.f;
    }
    if (t > first) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) hp[i] = to_float(x[(size_t)(t - 1) * ldx + c0 + i]);
    } else if (t < end) {
        const int slot = state_slots[s];
        if (slot >= 0 && slot < num_slots) {
            float* sp = prev + (size_t)slot * prev_stride + c0;
#pragma unroll
            for (int i = 0; i < VEC; ++i) hp[i] = sp[i];
#pragma unroll
            for (int i = 0; i < VEC; ++i) sp[i] = to_float(x[(size_t)(end - 1) * ldx + c0 + i]);
        }
    }
    for (int m = 0; m < n; ++m) {
        const float* mv = mu + (size_t)m * w + c0;
        T* o = out + ((size_t)m * tokens + t) * w + c0;
        float y[VEC];
#pragma unroll
        for (int i = 0; i < VEC; ++i) y[i] = h[i] + (hp[i] - h[i]) * mv[i];
        tm_store<T, VEC>(o, y);
    }
}

template <typename T>
static int launch_embed_bigram(const int* ids, const int* cu_q, const int* seq_of_token, const int* state_slots,
                               int* state, long long state_stride, int num_slots, const T* table, int vocab,
                               const T* pairs, long long buckets, long long mul_prev, long long mul_cur, float* out,
                               T* copy, int ldc, int T_, int h, cudaStream_t st) {
    if (T_ <= 0) return 0;
    if (h <= 0 || vocab <= 0 || buckets <= 0 || state == nullptr || state_stride < 1 || num_slots <= 0 ||
        pairs == nullptr || (copy != nullptr && ldc < h))
        return SLB_ERR_BAD_ARG;
    const bool vec = h % 4 == 0 && ldc % 4 == 0 &&
                     (((uintptr_t)table | (uintptr_t)pairs | (uintptr_t)out | (uintptr_t)copy) & 15) == 0;
    return slb_launch(vec ? embed_bigram_kernel<T, 4> : embed_bigram_kernel<T, 1>, dim3(T_), dim3(h >= 1024 ? 256 : 128),
                      0, st, ids, cu_q, seq_of_token,
                      state_slots, state, state_stride, num_slots, table, vocab, pairs, buckets, mul_prev, mul_cur,
                      out, copy, ldc, h);
}

template <typename T>
static int launch_token_mix(const T* x, int ldx, const float* mu, int n, float* prev, long long prev_stride,
                            int num_slots, const int* cu_q, const int* seq_of_token, const int* state_slots, T* out,
                            int w, int tokens, cudaStream_t st) {
    if (tokens <= 0) return 0;
    if (w <= 0 || ldx < w || n < 1 || n > TM_MAX || prev == nullptr || prev_stride < w || num_slots <= 0)
        return SLB_ERR_BAD_ARG;
    if (tokens > 65535) return SLB_ERR_TOO_LARGE;
    const bool vec = w % 4 == 0 && ((uintptr_t)out & 15) == 0;
    const int vecs = vec ? w / 4 : w;
    const int threads = vecs >= 256 ? 256 : (vecs + 31) / 32 * 32;
    const dim3 grid((vecs + threads - 1) / threads, tokens);
    if (vec)
        return slb_launch(token_mix_kernel<T, 4>, grid, dim3(threads), 0, st, x, ldx, mu, n, prev, prev_stride,
                          num_slots, cu_q, seq_of_token, state_slots, out, w, tokens);
    return slb_launch(token_mix_kernel<T, 1>, grid, dim3(threads), 0, st, x, ldx, mu, n, prev, prev_stride, num_slots,
                      cu_q, seq_of_token, state_slots, out, w, tokens);
}

extern "C" {
int slb_token_mix_max() { return TM_MAX; }
int slb_embed_bigram_f32(const int* ids, const int* cu_q, const int* seq_of_token, const int* state_slots, int* state,
                         long long state_stride, int num_slots, const float* table, int vocab, const float* pairs,
                         long long buckets, long long mul_prev, long long mul_cur, float* out, float* copy, int ldc,
                         int T, int h, cudaStream_t st) {
    return launch_embed_bigram<float>(ids, cu_q, seq_of_token, state_slots, state, state_stride, num_slots, table,
                                      vocab, pairs, buckets, mul_prev, mul_cur, out, copy, ldc, T, h, st);
}
int slb_embed_bigram_bf16(const int* ids, const int* cu_q, const int* seq_of_token, const int* state_slots, int* state,
                          long long state_stride, int num_slots, const bf16* table, int vocab, const bf16* pairs,
                          long long buckets, long long mul_prev, long long mul_cur, float* out, bf16* copy, int ldc,
                          int T, int h, cudaStream_t st) {
    return launch_embed_bigram<bf16>(ids, cu_q, seq_of_token, state_slots, state, state_stride, num_slots, table,
                                     vocab, pairs, buckets, mul_prev, mul_cur, out, copy, ldc, T, h, st);
}
int slb_token_mix_f32(const float* x, int ldx, const float* mu, int n, float* prev, long long prev_stride,
                      int num_slots, const int* cu_q, const int* seq_of_token, const int* state_slots, float* out,
                      int w, int tokens, cudaStream_t st) {
    return launch_token_mix<float>(x, ldx, mu, n, prev, prev_stride, num_slots, cu_q, seq_of_token, state_slots, out,
                                   w, tokens, st);
}
int slb_token_mix_bf16(const bf16* x, int ldx, const float* mu, int n, float* prev, long long prev_stride,
                       int num_slots, const int* cu_q, const int* seq_of_token, const int* state_slots, bf16* out,
                       int w, int tokens, cudaStream_t st) {
    return launch_token_mix<bf16>(x, ldx, mu, n, prev, prev_stride, num_slots, cu_q, seq_of_token, state_slots, out,
                                  w, tokens, st);
}
}
