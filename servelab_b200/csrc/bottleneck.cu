// The second product of a bottleneck, out = tanh(low) W^T (+ bias) with float32 results, for bfloat16
// rows and weights: mma.sync on tiles of 64 tokens x 64 outputs (128
// where there are many tokens: tanh is formed again for every tile of outputs).  tanh is formed in float32 and enters
// the product as two bfloat16 numbers (its value to 16 bits), so nothing of it is lost to the operand
// type; the sums are float32.  Any sizes; `low` may be columns of a larger projection.  A row of the
// result does not depend on the other rows of the batch.
#include "mma_util.cuh"

#define BN_M 64
#define BN_K 64
#define BN_LD (BN_K + 8)

template <int BN_N>
__global__ void __launch_bounds__(128) tanh_linear_mma_kernel(
    const bf16* __restrict__ A, int lda, const bf16* __restrict__ W, int ldw, float* __restrict__ C, int ldc,
    const float* __restrict__ bias, int M, int N, int K, int vec_a, int vec_w) {
    __shared__ __align__(16) bf16 Ah[BN_M][BN_LD], Al[BN_M][BN_LD], Ws[BN_N][BN_LD];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int m0 = blockIdx.y * BN_M, n0 = blockIdx.x * BN_N;
    pdl_launch_dependents();
    float acc[BN_N / 8][4] = {};
    for (int k0 = 0; k0 < K; k0 += BN_K) {
        // 16 bytes a thread: eight threads a row (weights: before the wait for the preceding kernel)
#pragma unroll
        for (int i = 0; i < BN_N / 16; ++i) {
            const int row = i * 16 + (tid >> 3), kk = (tid & 7) * 8;
            const int gn = n0 + row, gk = k0 + kk;
            uint4 v = make_uint4(0, 0, 0, 0);
            if (gn < N && gk < K) {
                const bf16* p = W + (size_t)gn * ldw + gk;
                if (vec_w) {
                    v = *reinterpret_cast<const uint4*>(p);
                } else {
                    bf16* e = reinterpret_cast<bf16*>(&v);
                    for (int j = 0; j < 8 && gk + j < K; ++j) e[j] = p[j];
                }
            }
            *reinterpret_cast<uint4*>(&Ws[row][kk]) = v;
        }
        if (k0 == 0) pdl_wait();
#pragma unroll
        for (int i = 0; i < BN_M / 16; ++i) {
            const int row = i * 16 + (tid >> 3), kk = (tid & 7) * 8;
            const int gm = m0 + row, gk = k0 + kk;
            uint4 v = make_uint4(0, 0, 0, 0), hi = v, lo = v;
            if (gm < M && gk < K) {
                const bf16* p = A + (size_t)gm * lda + gk;
                bf16* e = reinterpret_cast<bf16*>(&v);
                if (vec_a) v = *reinterpret_cast<const uint4*>(p);
                else
                    for (int j = 0; j < 8 && gk + j < K; ++j) e[j] = p[j];
                bf16* eh = reinterpret_cast<bf16*>(&hi);
                bf16* el = reinterpret_cast<bf16*>(&lo);
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    const float x = tanhf(__bfloat162float(e[j]));
                    eh[j] = __float2bfloat16_rn(x);
                    el[j] = __float2bfloat16_rn(x - __bfloat162float(eh[j]));
                }
            }
            *reinterpret_cast<uint4*>(&Ah[row][kk]) = hi;
            *reinterpret_cast<uint4*>(&Al[row][kk]) = lo;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < BN_K; kk += 16) {
            unsigned ah[4], al[4];
            slb_mma::ldmatrix_x4(ah, &Ah[warp * 16 + (lane & 15)][kk + (lane >> 4) * 8]);
            slb_mma::ldmatrix_x4(al, &Al[warp * 16 + (lane & 15)][kk + (lane >> 4) * 8]);
#pragma unroll
            for (int jp = 0; jp < BN_N / 16; ++jp) {
                unsigned b[4];
                slb_mma::ldmatrix_x4(b, &Ws[jp * 16 + (lane >> 4) * 8 + (lane & 7)][kk + ((lane >> 3) & 1) * 8]);
                slb_mma::mma_bf16(acc[2 * jp], al, b[0], b[1]);
                slb_mma::mma_bf16(acc[2 * jp + 1], al, b[2], b[3]);
                slb_mma::mma_bf16(acc[2 * jp], ah, b[0], b[1]);
                slb_mma::mma_bf16(acc[2 * jp + 1], ah, b[2], b[3]);
            }
        }
        __syncthreads();
    }
    const bool pairs = (ldc & 1) == 0 && ((uintptr_t)C & 7) == 0;
#pragma unroll
    for (int j = 0; j < BN_N / 8; ++j) {
        const int gn = n0 + j * 8 + (lane & 3) * 2;
        if (gn >= N) continue;
        const float b0 = bias != nullptr ? bias[gn] : 0.f, b1 = bias != nullptr && gn + 1 < N ? bias[gn + 1] : 0.f;
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int gm = m0 + warp * 16 + (lane >> 2) + r * 8;
            if (gm >= M) continue;
            float* o = C + (size_t)gm * ldc + gn;
            const float x = acc[j][2 * r] + b0, y = acc[j][2 * r + 1] + b1;
            if (pairs && gn + 1 < N) *reinterpret_cast<float2*>(o) = make_float2(x, y);
            else {
                o[0] = x;
                if (gn + 1 < N) o[1] = y;
            }
        }
    }
}

extern "C" int slb_tanh_linear_bf16(const bf16* A, int lda, const bf16* W, int ldw, float* C, int ldc,
                                    const float* bias, int M, int N, int K, cudaStream_t st) {
    if (M <= 0 || N <= 0) return 0;
    if (K <= 0 || lda < K || ldw < K || ldc < N) return SLB_ERR_BAD_ARG;
    const int gy = (M + BN_M - 1) / BN_M;
    if (gy > 65535) return SLB_ERR_TOO_LARGE;
    const int vec_a = K % 8 == 0 && lda % 8 == 0 && ((uintptr_t)A & 15) == 0;
    const int vec_w = K % 8 == 0 && ldw % 8 == 0 && ((uintptr_t)W & 15) == 0;
    if (M >= 512 && N > 64)
        return slb_launch(tanh_linear_mma_kernel<128>, dim3((N + 127) / 128, gy), dim3(128), 0, st, A, lda, W, ldw, C,
                          ldc, bias, M, N, K, vec_a, vec_w);
    return slb_launch(tanh_linear_mma_kernel<64>, dim3((N + 63) / 64, gy), dim3(128), 0, st, A, lda, W, ldw, C, ldc,
                      bias, M, N, K, vec_a, vec_w);
}
