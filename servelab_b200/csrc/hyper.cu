// Kernels around a residual that is kept as several parallel streams (hyper-connections), the
// RMS norm of an embedding, and the norm + gate that follows a head-wise mixer.
//
//   embed_norm_streams   out[t][s][:] = rmsnorm(table[ids[t]]) * w for s = 0..n-1 (w null: the
//                        embedding itself), float32: gather, norm and the copies in one pass.
//   hyper_mix_norm       with X [T][n][w] the float32 streams: an update y [T][w] that a sublayer
//                        left is folded in, X_t <- sum_s M[s][t] X_s + b[t] y (all streams at once
//                        from the old ones; M indexed [from][to]), then the next reader's input
//                        u = sum_s a[s] X_s (a null: the plain sum) is RMS-normed with a weight
//                        (null: u itself) into rows of the compute dtype.  With a row selection
//                        only those rows are produced and X is left as it is.  Each step optional.
//   group_norm_gate      y = x / sqrt(mean_group(x^2) + eps) * w * factor * act(gate) over groups of
//                        neighbouring elements (a head, or the whole row), where x is a float32 row
//                        or the difference a_1 - lambda a_2 of two maps stored side by side
//                        ([group][2][size]); w and gate optional; act: sigmoid or SiLU.
//
// All arithmetic float32; sums over a row run in an order that depends only on the row's size.
#include "common.cuh"

#define HY_MAX_STREAMS 8

template <typename T>
__global__ void __launch_bounds__(256) embed_norm_streams_kernel(
    const int* __restrict__ ids, const T* __restrict__ table, const float* __restrict__ w, float eps,
    float* __restrict__ out, int n, int h, int vocab) {
    __shared__ float scratch[33];
    pdl_wait();
    pdl_launch_dependents();
    const int t = blockIdx.x;
    const int id = ids[t];
    const bool ok = id >= 0 && id < vocab;
    const T* row = table + (size_t)(ok ? id : 0) * h;
    float rstd = 1.f;
    if (w != nullptr) {
        float ss = 0.f;
        for (int c = threadIdx.x; c < h; c += blockDim.x) {
            const float x = ok ? to_float(row[c]) : 0.f;
            ss += x * x;
        }
        ss = block_sum(ss, scratch);
        rstd = 1.0f / sqrtf(ss / (float)h + eps);
    }
    float* o = out + (size_t)t * n * h;
    for (int c = threadIdx.x; c < h; c += blockDim.x) {
        float x = ok ? to_float(row[c]) : 0.f;
        if (w != nullptr) x = x * rstd * w[c];
        for (int s = 0; s < n; ++s) o[(size_t)s * h + c] = x;
    }
}

template <typename T>
__global__ void __launch_bounds__(256) hyper_mix_norm_kernel(
    float* __restrict__ X, const T* __restrict__ y, int ldy, const float* __restrict__ M,
    const float* __restrict__ b, const float* __restrict__ a, const float* __restrict__ norm_w, float eps,
    T* __restrict__ out, int ldo, const int* __restrict__ row_map, int n, int w) {
    extern __shared__ float hy_u[];               // [w]: the reader's input before the norm
    __shared__ float scratch[33];
    __shared__ float sM[HY_MAX_STREAMS * HY_MAX_STREAMS], sb[HY_MAX_STREAMS], sa[HY_MAX_STREAMS];
    // (the small vectors are weights: read before the wait for the preceding kernel)
    for (int i = threadIdx.x; i < n * n; i += blockDim.x) sM[i] = M != nullptr ? M[i] : (i / n == i % n ? 1.f : 0.f);
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        sb[i] = b != nullptr ? b[i] : 1.f;
        sa[i] = a != nullptr ? a[i] : 1.f;
    }
    pdl_wait();
    pdl_launch_dependents();
    __syncthreads();
    const int r = blockIdx.x;
    const int t = row_map != nullptr ? row_map[r] : r;
    float* x = X + (size_t)t * n * w;
    const bool fold = y != nullptr;
    float ss = 0.f;
    for (int c = threadIdx.x; c < w; c += blockDim.x) {
        float old[HY_MAX_STREAMS];
#pragma unroll
        for (int s = 0; s < HY_MAX_STREAMS; ++s) old[s] = s < n ? x[(size_t)s * w + c] : 0.f;
        float u = 0.f;
        if (fold) {
            const float yv = to_float(y[(size_t)t * ldy + c]);
#pragma unroll
            for (int to = 0; to < HY_MAX_STREAMS; ++to) {
                if (to < n) {
                    float v = 0.f;
#pragma unroll
                    for (int s = 0; s < HY_MAX_STREAMS; ++s)
                        if (s < n) v = fmaf(sM[s * n + to], old[s], v);
                    v = fmaf(sb[to], yv, v);
                    if (row_map == nullptr) x[(size_t)to * w + c] = v;
                    u = fmaf(sa[to], v, u);
                }
            }
        } else {
#pragma unroll
            for (int s = 0; s < HY_MAX_STREAMS; ++s)
                if (s < n) u = fmaf(sa[s], old[s], u);
        }
        hy_u[c] = u;
        ss += u * u;
    }
    if (out == nullptr) return;
    float rstd = 1.f;
    if (norm_w != nullptr) {
        ss = block_sum(ss, scratch);
        rstd = 1.0f / sqrtf(ss / (float)w + eps);
    }
    T* o = out + (size_t)r * ldo;
    for (int c = threadIdx.x; c < w; c += blockDim.x)     // (a thread reads back what it wrote itself)
        o[c] = from_float<T>(norm_w != nullptr ? hy_u[c] * rstd * norm_w[c] : hy_u[c]);
}

// a warp a (token, group)
template <typename T>
__global__ void __launch_bounds__(128) group_norm_gate_kernel(
    const float* __restrict__ in, int ldi, int maps, const float* __restrict__ lam,
    const float* __restrict__ w, float eps, float factor, const T* __restrict__ gate, int ldg, int gate_act,
    T* __restrict__ out, int ldo, int T_, int groups, int size) {
    pdl_wait();
    pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long unit = (long long)blockIdx.x * 4 + warp;
    if (unit >= (long long)T_ * groups) return;
    const int t = (int)(unit / groups), g = (int)(unit - (long long)t * groups);
    const float* x1 = in + (size_t)t * ldi + (size_t)g * maps * size;
    const float* x2 = x1 + size;
    const float l = maps == 2 ? lam[0] : 0.f;
    float ss = 0.f;
    for (int c = lane; c < size; c += 32) {
        const float x = maps == 2 ? x1[c] - l * x2[c] : x1[c];
        ss += x * x;
    }
    ss = warp_sum(ss);
    const float rstd = factor / sqrtf(ss / (float)size + eps);
    for (int c = lane; c < size; c += 32) {
        float x = (maps == 2 ? x1[c] - l * x2[c] : x1[c]) * rstd;
        const int col = g * size + c;
        if (w != nullptr) x *= w[col];
        if (gate != nullptr) {
            const float z = to_float(gate[(size_t)t * ldg + col]);
            const float sg = 1.0f / (1.0f + expf(-z));
            x *= gate_act == 2 ? z * sg : sg;
        }
        out[(size_t)t * ldo + col] = from_float<T>(x);
    }
}

// The gate before the norm: v = x * act(gate), every one of `groups` equal parts of a row divided by its own root
// mean square, times a weight over the row and a factor.  A block a (token, part); x float32, float32 arithmetic;
// a thread keeps GGN_NV vectors of V elements in registers, longer parts are formed again.
#define GGN_THREADS 256
#define GGN_NV 4
__device__ __forceinline__ float gated_by(float x, float z, int gate_act) {
    const float sg = 1.0f / (1.0f + expf(-z));
    return x * (gate_act == 2 ? z * sg : sg);
}
__device__ __forceinline__ void ggn_load(const float* p, float (&v)[4]) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
}
__device__ __forceinline__ void ggn_load(const bf16* p, float (&v)[4]) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}
template <typename T> __device__ __forceinline__ void ggn_load(const T* p, float (&v)[1]) { v[0] = to_float(p[0]); }
__device__ __forceinline__ void ggn_store(float* p, const float (&v)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ void ggn_store(bf16* p, const float (&v)[4]) {
    __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<unsigned*>(&lo), *reinterpret_cast<unsigned*>(&hi));
}
template <typename T> __device__ __forceinline__ void ggn_store(T* p, const float (&v)[1]) { p[0] = from_float<T>(v[0]); }

template <typename T, int V>
__global__ void __launch_bounds__(GGN_THREADS) gate_group_norm_kernel(
    const float* __restrict__ x, int ldx, const T* __restrict__ gate, int ldg, int gate_act, const float* __restrict__ w,
    float eps, float factor, T* __restrict__ out, int ldo, int size) {
    __shared__ float scratch[33];
    pdl_wait();
    pdl_launch_dependents();
    const size_t t = blockIdx.x;
    const int c0 = blockIdx.y * size;
    const float* xr = x + t * ldx + c0;
    const T* gr = gate + t * ldg + c0;
    T* o = out + t * ldo + c0;
    float v[GGN_NV][V], z[GGN_NV][V];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < GGN_NV; ++j) {
        const int c = (threadIdx.x + j * blockDim.x) * V;
        if (c < size) {
            ggn_load(xr + c, v[j]);
            ggn_load(gr + c, z[j]);
        }
    }
#pragma unroll
    for (int j = 0; j < GGN_NV; ++j) {
        const int c = (threadIdx.x + j * blockDim.x) * V;
        if (c < size) {
#pragma unroll
            for (int e = 0; e < V; ++e) {
                v[j][e] = gated_by(v[j][e], z[j][e], gate_act);
                ss += v[j][e] * v[j][e];
            }
        }
    }
    for (int c = threadIdx.x + GGN_NV * V * blockDim.x; c < size; c += blockDim.x) {
        const float u = gated_by(xr[c], to_float(gr[c]), gate_act);
        ss += u * u;
    }
    const float rstd = factor / sqrtf(block_sum(ss, scratch) / (float)size + eps);
#pragma unroll
    for (int j = 0; j < GGN_NV; ++j) {
        const int c = (threadIdx.x + j * blockDim.x) * V;
        if (c < size) {
            float wv[V];
            if (w != nullptr) ggn_load(w + c0 + c, wv);
#pragma unroll
            for (int e = 0; e < V; ++e) v[j][e] *= rstd * (w != nullptr ? wv[e] : 1.f);
            ggn_store(o + c, v[j]);
        }
    }
    for (int c = threadIdx.x + GGN_NV * V * blockDim.x; c < size; c += blockDim.x)
        o[c] = from_float<T>(gated_by(xr[c], to_float(gr[c]), gate_act) * rstd * (w != nullptr ? w[c0 + c] : 1.f));
}

template <typename T>
static int launch_gate_group_norm(const float* x, int ldx, const T* gate, int ldg, int gate_act, const float* w,
                                  float eps, float factor, T* out, int ldo, int T_, int groups, int size,
                                  cudaStream_t st) {
    if (T_ <= 0) return 0;
    if (groups <= 0 || groups > 65535 || size <= 0 || gate == nullptr || gate_act < 1 || gate_act > 2 ||
        ldx < groups * size || ldg < groups * size || ldo < groups * size)
        return SLB_ERR_BAD_ARG;
    const uintptr_t half = (uintptr_t)gate | (uintptr_t)out;
    const bool vec = ((size | ldx | ldg | ldo) & 3) == 0 && (((uintptr_t)x | (uintptr_t)w) & 15) == 0 &&
                     (half & (4 * sizeof(T) - 1)) == 0;
    const int units = vec ? size / 4 : size;
    int threads = (units + 31) / 32 * 32;
    threads = threads > GGN_THREADS ? GGN_THREADS : threads;
    if (vec)
        return slb_launch(gate_group_norm_kernel<T, 4>, dim3(T_, groups), dim3(threads), 0, st, x, ldx, gate, ldg,
                          gate_act, w, eps, factor, out, ldo, size);
    return slb_launch(gate_group_norm_kernel<T, 1>, dim3(T_, groups), dim3(threads), 0, st, x, ldx, gate, ldg, gate_act,
                      w, eps, factor, out, ldo, size);
}

template <typename T>
static int launch_hyper_mix_norm(float* X, const T* y, int ldy, const float* M, const float* b, const float* a,
                                 const float* norm_w, float eps, T* out, int ldo, const int* row_map, int rows,
                                 int n, int w, cudaStream_t st) {
    if (rows <= 0) return 0;
    if (n <= 0 || w <= 0 || (y != nullptr && ldy < w) || (out != nullptr && ldo < w)) return SLB_ERR_BAD_ARG;
    if (n > HY_MAX_STREAMS || (size_t)w * sizeof(float) > 200 * 1024) return SLB_ERR_TOO_LARGE;
    const size_t smem = (size_t)w * sizeof(float);
    static unsigned long long configured = 0;
    if (smem > 48 * 1024) {
        const int rc = slb_configure(&configured, hyper_mix_norm_kernel<T>, 200 * 1024);
        if (rc != 0) return rc;
    }
    int threads = ((w + 3) / 4 + 31) / 32 * 32;
    threads = threads < 32 ? 32 : (threads > 256 ? 256 : threads);
    return slb_launch(hyper_mix_norm_kernel<T>, dim3(rows), dim3(threads), smem, st, X, y, ldy, M, b, a, norm_w,
                      eps, out, ldo, row_map, n, w);
}

template <typename T>
static int launch_group_norm_gate(const float* in, int ldi, int maps, const float* lam, const float* w, float eps,
                                  float factor, const T* gate, int ldg, int gate_act, T* out, int ldo, int T_,
                                  int groups, int size, cudaStream_t st) {
    if (T_ <= 0) return 0;
    if (groups <= 0 || size <= 0 || (maps != 1 && maps != 2) || (maps == 2 && lam == nullptr) ||
        gate_act < 0 || gate_act > 2 || (gate != nullptr && gate_act == 0))
        return SLB_ERR_BAD_ARG;
    const long long units = (long long)T_ * groups;
    if ((units + 3) / 4 > 2147483647LL) return SLB_ERR_TOO_LARGE;
    return slb_launch(group_norm_gate_kernel<T>, dim3((unsigned)((units + 3) / 4)), dim3(128), 0, st, in, ldi, maps,
                      lam, w, eps, factor, gate, ldg, gate_act, out, ldo, T_, groups, size);
}

// out[t] = x[t] / sqrt(mean(x[t]^2) + eps) * w over the first n columns of every row (a latent
// inside a wider projection); a block a row, float32 arithmetic.
template <typename T>
__global__ void __launch_bounds__(256) rms_norm_rows_kernel(const T* __restrict__ x, int ldx,
                                                            const float* __restrict__ w, float eps,
                                                            T* __restrict__ out, int ldo, int n) {
    __shared__ float scratch[33];
    pdl_wait();
    pdl_launch_dependents();
    const T* row = x + (size_t)blockIdx.x * ldx;
    float ss = 0.f;
    for (int c = threadIdx.x; c < n; c += blockDim.x) {
        const float v = to_float(row[c]);
        ss += v * v;
    }
    ss = block_sum(ss, scratch);
    const float rstd = 1.0f / sqrtf(ss / (float)n + eps);
    for (int c = threadIdx.x; c < n; c += blockDim.x)
        out[(size_t)blockIdx.x * ldo + c] = from_float<T>(to_float(row[c]) * rstd * (w != nullptr ? w[c] : 1.f));
}

// out[t] = factor * (a[t] / rms(a[t]) * wa + b[t] / rms(b[t]) * wb): the results of two branches
// that read the same input, each RMS-normed over the row with a weight of its own, summed.
// a and b float32 [T, n]; a block a row; float32 arithmetic.
template <typename T>
__global__ void __launch_bounds__(256) norm_sum2_kernel(const float* __restrict__ a, int lda,
                                                        const float* __restrict__ b, int ldb,
                                                        const float* __restrict__ wa, const float* __restrict__ wb,
                                                        float eps, float factor, T* __restrict__ out, int ldo, int n) {
    __shared__ float scratch[33];
    pdl_wait();
    pdl_launch_dependents();
    const float* ra = a + (size_t)blockIdx.x * lda;
    const float* rb = b + (size_t)blockIdx.x * ldb;
    float sa = 0.f, sb = 0.f;
    for (int c = threadIdx.x; c < n; c += blockDim.x) {
        sa += ra[c] * ra[c];
        sb += rb[c] * rb[c];
    }
    sa = block_sum(sa, scratch);
    sb = block_sum(sb, scratch);
    const float fa = 1.0f / sqrtf(sa / (float)n + eps), fb = 1.0f / sqrtf(sb / (float)n + eps);
    for (int c = threadIdx.x; c < n; c += blockDim.x)
        out[(size_t)blockIdx.x * ldo + c] = from_float<T>(factor * (ra[c] * fa * wa[c] + rb[c] * fb * wb[c]));
}

extern "C" {
int slb_rms_norm_rows_f32(const float* x, int ldx, const float* w, float eps, float* out, int ldo, int T, int n,
                          cudaStream_t st) {
    if (T <= 0) return 0;
    if (n <= 0 || ldx < n || ldo < n) return SLB_ERR_BAD_ARG;
    return slb_launch(rms_norm_rows_kernel<float>, dim3(T), dim3(n >= 1024 ? 256 : 128), 0, st, x, ldx, w, eps, out,
                      ldo, n);
}
int slb_rms_norm_rows_bf16(const bf16* x, int ldx, const float* w, float eps, bf16* out, int ldo, int T, int n,
                           cudaStream_t st) {
    if (T <= 0) return 0;
    if (n <= 0 || ldx < n || ldo < n) return SLB_ERR_BAD_ARG;
    return slb_launch(rms_norm_rows_kernel<bf16>, dim3(T), dim3(n >= 1024 ? 256 : 128), 0, st, x, ldx, w, eps, out,
                      ldo, n);
}
int slb_norm_sum2_f32(const float* a, int lda, const float* b, int ldb, const float* wa, const float* wb, float eps,
                      float factor, float* out, int ldo, int T, int n, cudaStream_t st) {
    if (T <= 0) return 0;
    if (n <= 0 || lda < n || ldb < n || ldo < n || wa == nullptr || wb == nullptr) return SLB_ERR_BAD_ARG;
    return slb_launch(norm_sum2_kernel<float>, dim3(T), dim3(256), 0, st, a, lda, b, ldb, wa, wb, eps, factor, out,
                      ldo, n);
}
int slb_norm_sum2_bf16(const float* a, int lda, const float* b, int ldb, const float* wa, const float* wb, float eps,
                       float factor, bf16* out, int ldo, int T, int n, cudaStream_t st) {
    if (T <= 0) return 0;
    if (n <= 0 || lda < n || ldb < n || ldo < n || wa == nullptr || wb == nullptr) return SLB_ERR_BAD_ARG;
    return slb_launch(norm_sum2_kernel<bf16>, dim3(T), dim3(256), 0, st, a, lda, b, ldb, wa, wb, eps, factor, out,
                      ldo, n);
}
int slb_hyper_max_streams() { return HY_MAX_STREAMS; }
int slb_embed_norm_streams_f32(const int* ids, const float* table, const float* w, float eps, float* out, int T,
                               int n, int h, int vocab, cudaStream_t st) {
    if (T <= 0) return 0;
    if (n <= 0 || h <= 0 || vocab <= 0) return SLB_ERR_BAD_ARG;
    return slb_launch(embed_norm_streams_kernel<float>, dim3(T), dim3(256), 0, st, ids, table, w, eps, out, n, h, vocab);
}
int slb_embed_norm_streams_bf16(const int* ids, const bf16* table, const float* w, float eps, float* out, int T,
                                int n, int h, int vocab, cudaStream_t st) {
    if (T <= 0) return 0;
    if (n <= 0 || h <= 0 || vocab <= 0) return SLB_ERR_BAD_ARG;
    return slb_launch(embed_norm_streams_kernel<bf16>, dim3(T), dim3(256), 0, st, ids, table, w, eps, out, n, h, vocab);
}
int slb_hyper_mix_norm_f32(float* X, const float* y, int ldy, const float* M, const float* b, const float* a,
                           const float* norm_w, float eps, float* out, int ldo, const int* row_map, int rows, int n,
                           int w, cudaStream_t st) {
    return launch_hyper_mix_norm<float>(X, y, ldy, M, b, a, norm_w, eps, out, ldo, row_map, rows, n, w, st);
}
int slb_hyper_mix_norm_bf16(float* X, const bf16* y, int ldy, const float* M, const float* b, const float* a,
                            const float* norm_w, float eps, bf16* out, int ldo, const int* row_map, int rows, int n,
                            int w, cudaStream_t st) {
    return launch_hyper_mix_norm<bf16>(X, y, ldy, M, b, a, norm_w, eps, out, ldo, row_map, rows, n, w, st);
}
int slb_gate_group_norm_f32(const float* x, int ldx, const float* gate, int ldg, int gate_act, const float* w, float eps,
                            float factor, float* out, int ldo, int T, int groups, int size, cudaStream_t st) {
    return launch_gate_group_norm<float>(x, ldx, gate, ldg, gate_act, w, eps, factor, out, ldo, T, groups, size, st);
}
int slb_gate_group_norm_bf16(const float* x, int ldx, const bf16* gate, int ldg, int gate_act, const float* w, float eps,
                             float factor, bf16* out, int ldo, int T, int groups, int size, cudaStream_t st) {
    return launch_gate_group_norm<bf16>(x, ldx, gate, ldg, gate_act, w, eps, factor, out, ldo, T, groups, size, st);
}
int slb_group_norm_gate_f32(const float* in, int ldi, int maps, const float* lam, const float* w, float eps,
                            float factor, const float* gate, int ldg, int gate_act, float* out, int ldo, int T,
                            int groups, int size, cudaStream_t st) {
    return launch_group_norm_gate<float>(in, ldi, maps, lam, w, eps, factor, gate, ldg, gate_act, out, ldo, T, groups,
                                         size, st);
}
int slb_group_norm_gate_bf16(const float* in, int ldi, int maps, const float* lam, const float* w, float eps,
                             float factor, const bf16* gate, int ldg, int gate_act, bf16* out, int ldo, int T,
                             int groups, int size, cudaStream_t st) {
    return launch_group_norm_gate<bf16>(in, ldi, maps, lam, w, eps, factor, gate, ldg, gate_act, out, ldo, T, groups,
                                        size, st);
}
}
