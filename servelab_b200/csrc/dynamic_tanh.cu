// Dynamic Tanh norm fused with the residual add around it.
//
// y = tanh(alpha * x) * w + b per element (alpha a learned scalar): no mean, no variance,
// no root mean square, so a row needs no reduction and the kernel is a plain elementwise
// pass over the float32 residual stream.  One launch does up to three things for a row:
//
//   d      = post != null ? tanh(post_alpha * delta) * post_w + post_b : delta
//            (the norm on a sublayer's RESULT, applied before the result is added)
//   resid += d                     (in place, float32; skipped when rows are selected)
//   out    = tanh(alpha * resid) * w + b   (the norm on the NEXT sublayer's input)
//
// All arithmetic is float32; `delta` and `out` have the compute type T.  The scalars are
// read from device memory, so the launch takes no value from the host.
//
// dyt_parallel serves a block whose two sublayers read the same stream, each behind a norm of
// its own, and whose first one may read its input mixed with the previous token's:
//
//   x    = resid + delta1 + delta2 + row          (each term optional; row is one vector for all tokens)
//   n1   = tanh(a1 x) w1 + b1;   out1 = n1 + (n1_previous - n1) * shift      (shift optional)
//   out2 = tanh(a2 x) w2 + b2                                                (optional)
//
// x goes to a buffer of its own, not over resid: the thread of the next token forms this token's
// n1 again from resid and the deltas (nothing is reduced over a row, so that is cheaper than a
// second pass).  n1_previous of the first token of a request's portion comes from the request's
// state record, and the thread that reads it there also leaves n1 of the portion's last token in
// it: one launch, no other thread touches that element of the record.  Tokens that belong to no
// request (the padding of a captured step) leave every record alone.
#include "common.cuh"

struct DytParallelArgs {
    const float* resid; int ldr;
    const void* d1; int ldd1; const void* d2; int ldd2; int d_is_f32;
    const float* row;
    float* resid_out; int ldx;
    const float* alpha1; const float* w1; const float* b1; void* out1; int ldo1;
    const float* shift;
    const float* alpha2; const float* w2; const float* b2; void* out2; int ldo2;
    float* prev; long long prev_stride; int num_slots;      // [slots][>= dim] float32
    const int* cu_q; const int* seq_of_token; const int* state_slots;
    const int* row_map;                                     // only these rows (no shift, no resid_out)
    int rows, dim;
};

template <typename T, int VEC>
__device__ __forceinline__ void dp_load_x(const DytParallelArgs& a, size_t t, int c0, float (&x)[VEC]) {
    const float* rp = a.resid + t * a.ldr + c0;
    if constexpr (VEC == 4) {
        const float4 v = *reinterpret_cast<const float4*>(rp);
        x[0] = v.x; x[1] = v.y; x[2] = v.z; x[3] = v.w;
    } else {
        x[0] = rp[0];
    }
    const void* ds[2] = {a.d1, a.d2};
    const int ld[2] = {a.ldd1, a.ldd2};
#pragma unroll
    for (int k = 0; k < 2; ++k) {
        if (ds[k] == nullptr) continue;
        if (a.d_is_f32 >> k & 1) {
            const float* dp = reinterpret_cast<const float*>(ds[k]) + t * ld[k] + c0;
            if constexpr (VEC == 4) {
                const float4 v = *reinterpret_cast<const float4*>(dp);
                x[0] += v.x; x[1] += v.y; x[2] += v.z; x[3] += v.w;
            } else {
                x[0] += dp[0];
            }
        } else {
            const T* dp = reinterpret_cast<const T*>(ds[k]) + t * ld[k] + c0;
            if constexpr (VEC == 4 && sizeof(T) == 2) {
                const uint2 u = *reinterpret_cast<const uint2*>(dp);
                const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
                const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
                x[0] += lo.x; x[1] += lo.y; x[2] += hi.x; x[3] += hi.y;
            } else {
#pragma unroll
                for (int i = 0; i < VEC; ++i) x[i] += to_float(dp[i]);
            }
        }
    }
    if (a.row != nullptr) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) x[i] += a.row[c0 + i];
    }
}

template <typename T, int VEC>
__device__ __forceinline__ void dp_store(T* p, const float (&v)[VEC]) {
    if constexpr (VEC == 4 && sizeof(T) == 2) {
        __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<unsigned*>(&lo), *reinterpret_cast<unsigned*>(&hi));
    } else if constexpr (VEC == 4) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    } else {
        p[0] = from_float<T>(v[0]);
    }
}

// A thread owns VEC columns of R neighbouring tokens: n1 of a token is carried to the next one.
template <typename T, int VEC, int R>
__global__ void __launch_bounds__(256) dyt_parallel_kernel(const DytParallelArgs a) {
    const int c0 = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
    if (c0 >= a.dim) return;
    // (weights: before the wait for the preceding kernel)
    const float al1 = a.alpha1 != nullptr ? *a.alpha1 : 0.f, al2 = a.alpha2 != nullptr ? *a.alpha2 : 0.f;
    float w1[VEC], b1[VEC], w2[VEC], b2[VEC], sh[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
        w1[i] = a.out1 != nullptr ? a.w1[c0 + i] : 0.f;
        b1[i] = a.out1 != nullptr ? a.b1[c0 + i] : 0.f;
        w2[i] = a.out2 != nullptr ? a.w2[c0 + i] : 0.f;
        b2[i] = a.out2 != nullptr ? a.b2[c0 + i] : 0.f;
        sh[i] = a.shift != nullptr ? a.shift[c0 + i] : 0.f;
    }
    pdl_launch_dependents();
    pdl_wait();
    float carry[VEC];
    bool carried = false;
#pragma unroll
    for (int r = 0; r < R; ++r) {
        const int row = blockIdx.y * R + r;
        if (row >= a.rows) break;
        const int t = a.row_map != nullptr ? a.row_map[row] : row;
        float x[VEC], n1[VEC], y[VEC];
        dp_load_x<T, VEC>(a, t, c0, x);
        if (a.resid_out != nullptr) dp_store<float, VEC>(a.resid_out + (size_t)t * a.ldx + c0, x);
        if (a.out1 != nullptr) {
#pragma unroll
            for (int i = 0; i < VEC; ++i) y[i] = n1[i] = tanhf(al1 * x[i]) * w1[i] + b1[i];
            if (a.shift != nullptr) {
                const int s = a.seq_of_token[t];
                const int first = a.cu_q[s], end = a.cu_q[s + 1];
                float hp[VEC];
                if (t > first) {
                    if (carried) {
#pragma unroll
                        for (int i = 0; i < VEC; ++i) hp[i] = carry[i];
                    } else {
                        float xp[VEC];
                        dp_load_x<T, VEC>(a, t - 1, c0, xp);
#pragma unroll
                        for (int i = 0; i < VEC; ++i) hp[i] = tanhf(al1 * xp[i]) * w1[i] + b1[i];
                    }
                } else {
                    const int slot = t < end ? a.state_slots[s] : -1;
#pragma unroll
                    for (int i = 0; i < VEC; ++i) hp[i] = 0.f;
                    if (slot >= 0 && slot < a.num_slots) {
                        float* sp = a.prev + (size_t)slot * a.prev_stride + c0;
#pragma unroll
                        for (int i = 0; i < VEC; ++i) hp[i] = sp[i];
                        float last[VEC];
                        if (end - 1 == t) {
#pragma unroll
                            for (int i = 0; i < VEC; ++i) last[i] = n1[i];
                        } else {
                            dp_load_x<T, VEC>(a, end - 1, c0, last);
#pragma unroll
                            for (int i = 0; i < VEC; ++i) last[i] = tanhf(al1 * last[i]) * w1[i] + b1[i];
                        }
#pragma unroll
                        for (int i = 0; i < VEC; ++i) sp[i] = last[i];
                    }
                }
#pragma unroll
                for (int i = 0; i < VEC; ++i) {
                    y[i] = n1[i] + (hp[i] - n1[i]) * sh[i];
                    carry[i] = n1[i];
                }
                carried = true;
            }
            dp_store<T, VEC>(reinterpret_cast<T*>(a.out1) + (size_t)row * a.ldo1 + c0, y);
        }
        if (a.out2 != nullptr) {
#pragma unroll
            for (int i = 0; i < VEC; ++i) y[i] = tanhf(al2 * x[i]) * w2[i] + b2[i];
            dp_store<T, VEC>(reinterpret_cast<T*>(a.out2) + (size_t)row * a.ldo2 + c0, y);
        }
    }
}

template <typename T>
static int launch_dyt_parallel(const DytParallelArgs& a, cudaStream_t st) {
    if (a.rows <= 0) return 0;
    if (a.dim <= 0 || a.resid == nullptr) return SLB_ERR_BAD_ARG;
    if (a.out1 != nullptr && (a.alpha1 == nullptr || a.w1 == nullptr || a.b1 == nullptr)) return SLB_ERR_BAD_ARG;
    if (a.out2 != nullptr && (a.alpha2 == nullptr || a.w2 == nullptr || a.b2 == nullptr)) return SLB_ERR_BAD_ARG;
    if (a.resid_out == a.resid) return SLB_ERR_BAD_ARG;
    if (a.row_map != nullptr && (a.shift != nullptr || a.resid_out != nullptr)) return SLB_ERR_BAD_ARG;
    if (a.shift != nullptr && (a.out1 == nullptr || a.prev == nullptr || a.num_slots <= 0 || a.prev_stride < a.dim ||
                               a.cu_q == nullptr || a.seq_of_token == nullptr || a.state_slots == nullptr))
        return SLB_ERR_BAD_ARG;
    const bool vec = a.dim % 4 == 0 && a.ldr % 4 == 0 && a.ldd1 % 4 == 0 && a.ldd2 % 4 == 0 && a.ldx % 4 == 0 &&
                     a.ldo1 % 4 == 0 && a.ldo2 % 4 == 0 &&
                     (((uintptr_t)a.resid | (uintptr_t)a.resid_out | (uintptr_t)a.d1 | (uintptr_t)a.d2 |
                       (uintptr_t)a.out1 | (uintptr_t)a.out2) & 15) == 0;
    const int vecs = vec ? a.dim / 4 : a.dim;
    const int threads = vecs >= 256 ? 256 : (vecs + 31) / 32 * 32;
    const bool many = a.rows >= 512;
    const int R = many ? 4 : 1;
    const dim3 grid((vecs + threads - 1) / threads, (a.rows + R - 1) / R);
    if (grid.y > 65535) return SLB_ERR_TOO_LARGE;
    if (vec)
        return many ? slb_launch(dyt_parallel_kernel<T, 4, 4>, grid, dim3(threads), 0, st, a)
                    : slb_launch(dyt_parallel_kernel<T, 4, 1>, grid, dim3(threads), 0, st, a);
    return many ? slb_launch(dyt_parallel_kernel<T, 1, 4>, grid, dim3(threads), 0, st, a)
                : slb_launch(dyt_parallel_kernel<T, 1, 1>, grid, dim3(threads), 0, st, a);
}

// out = resid + d1 + d2 + row (terms as above) in the compute type: the stream as the operand of a product.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) stream_rows_kernel(const DytParallelArgs a) {
    const int c0 = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
    pdl_launch_dependents();
    pdl_wait();
    if (c0 >= a.dim) return;
    float x[VEC];
    dp_load_x<T, VEC>(a, blockIdx.y, c0, x);
    dp_store<T, VEC>(reinterpret_cast<T*>(a.out1) + (size_t)blockIdx.y * a.ldo1 + c0, x);
}

template <typename T>
static int launch_stream_rows(const DytParallelArgs& a, cudaStream_t st) {
    if (a.rows <= 0) return 0;
    if (a.dim <= 0 || a.resid == nullptr || a.out1 == nullptr) return SLB_ERR_BAD_ARG;
    if (a.rows > 65535) return SLB_ERR_TOO_LARGE;
    const bool vec = a.dim % 4 == 0 && a.ldr % 4 == 0 && a.ldd1 % 4 == 0 && a.ldd2 % 4 == 0 && a.ldo1 % 4 == 0 &&
                     (((uintptr_t)a.resid | (uintptr_t)a.d1 | (uintptr_t)a.d2 | (uintptr_t)a.out1) & 15) == 0;
    const int vecs = vec ? a.dim / 4 : a.dim;
    const int threads = vecs >= 256 ? 256 : (vecs + 31) / 32 * 32;
    const dim3 grid((vecs + threads - 1) / threads, a.rows);
    return vec ? slb_launch(stream_rows_kernel<T, 4>, grid, dim3(threads), 0, st, a)
               : slb_launch(stream_rows_kernel<T, 1>, grid, dim3(threads), 0, st, a);
}

template <typename T, int VEC>
__global__ void __launch_bounds__(256) dyt_add_norm_kernel(
    float* __restrict__ resid, int ldr, const T* __restrict__ delta, int ldd,
    const float* __restrict__ post_alpha, const float* __restrict__ post_w,
    const float* __restrict__ post_b, const float* __restrict__ alpha,
    const float* __restrict__ w, const float* __restrict__ b, T* __restrict__ out, int ldo,
    const int* __restrict__ row_map, int dim) {
    const float pa = post_alpha != nullptr ? *post_alpha : 0.f;      // (weights: before the wait)
    const float a = alpha != nullptr ? *alpha : 0.f;
    pdl_launch_dependents();
    pdl_wait();
    const int r = blockIdx.y;
    const int src = row_map != nullptr ? row_map[r] : r;
    const int c0 = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
    if (c0 >= dim) return;
    float x[VEC];
    float* rp = resid + (size_t)src * ldr + c0;
    if constexpr (VEC == 4) {
        const float4 v = *reinterpret_cast<const float4*>(rp);
        x[0] = v.x; x[1] = v.y; x[2] = v.z; x[3] = v.w;
    } else {
        x[0] = rp[0];
    }
    if (delta != nullptr) {
        const T* dp = delta + (size_t)src * ldd + c0;
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            float d = to_float(dp[i]);
            if (post_alpha != nullptr) d = tanhf(pa * d) * post_w[c0 + i] + post_b[c0 + i];
            x[i] += d;
        }
        if (row_map == nullptr) {
            if constexpr (VEC == 4) *reinterpret_cast<float4*>(rp) = make_float4(x[0], x[1], x[2], x[3]);
            else rp[0] = x[0];
        }
    }
    if (out != nullptr) {
        T* op = out + (size_t)r * ldo + c0;
#pragma unroll
        for (int i = 0; i < VEC; ++i) op[i] = from_float<T>(tanhf(a * x[i]) * w[c0 + i] + b[c0 + i]);
    }
}

template <typename T>
static int launch_dyt(float* resid, int ldr, const T* delta, int ldd, const float* post_alpha,
                      const float* post_w, const float* post_b, const float* alpha, const float* w,
                      const float* b, T* out, int ldo, const int* row_map, int rows, int dim,
                      cudaStream_t st) {
    if (rows <= 0) return 0;
    if (dim <= 0 || resid == nullptr || rows > 65535 * 1024) return SLB_ERR_BAD_ARG;
    if (out != nullptr && (alpha == nullptr || w == nullptr || b == nullptr)) return SLB_ERR_BAD_ARG;
    if (post_alpha != nullptr && (post_w == nullptr || post_b == nullptr || delta == nullptr)) return SLB_ERR_BAD_ARG;
    if (rows > 65535) return SLB_ERR_TOO_LARGE;
    const bool vec = dim % 4 == 0 && ldr % 4 == 0 && ((uintptr_t)resid & 15) == 0;
    if (vec) {
        const dim3 grid((dim / 4 + 255) / 256, rows);
        return slb_launch(dyt_add_norm_kernel<T, 4>, grid, dim3(256), 0, st, resid, ldr, delta, ldd,
                          post_alpha, post_w, post_b, alpha, w, b, out, ldo, row_map, dim);
    }
    const dim3 grid((dim + 255) / 256, rows);
    return slb_launch(dyt_add_norm_kernel<T, 1>, grid, dim3(256), 0, st, resid, ldr, delta, ldd,
                      post_alpha, post_w, post_b, alpha, w, b, out, ldo, row_map, dim);
}

extern "C" {
int slb_dyt_parallel_f32(const DytParallelArgs* a, cudaStream_t st) { return launch_dyt_parallel<float>(*a, st); }
int slb_dyt_parallel_bf16(const DytParallelArgs* a, cudaStream_t st) { return launch_dyt_parallel<bf16>(*a, st); }
int slb_stream_rows_f32(const DytParallelArgs* a, cudaStream_t st) { return launch_stream_rows<float>(*a, st); }
int slb_stream_rows_bf16(const DytParallelArgs* a, cudaStream_t st) { return launch_stream_rows<bf16>(*a, st); }
int slb_dyt_add_norm_f32(float* resid, int ldr, const float* delta, int ldd, const float* post_alpha,
                         const float* post_w, const float* post_b, const float* alpha, const float* w,
                         const float* b, float* out, int ldo, const int* row_map, int rows, int dim,
                         cudaStream_t st) {
    return launch_dyt<float>(resid, ldr, delta, ldd, post_alpha, post_w, post_b, alpha, w, b, out, ldo,
                             row_map, rows, dim, st);
}
int slb_dyt_add_norm_bf16(float* resid, int ldr, const bf16* delta, int ldd, const float* post_alpha,
                          const float* post_w, const float* post_b, const float* alpha, const float* w,
                          const float* b, bf16* out, int ldo, const int* row_map, int rows, int dim,
                          cudaStream_t st) {
    return launch_dyt<bf16>(resid, ldr, delta, ldd, post_alpha, post_w, post_b, alpha, w, b, out, ldo,
                            row_map, rows, dim, st);
}
}
