// The selective state space (state_space.cu) for steps that bring portions of prompts, in its chunked form on
// the tensor cores (bf16 mma.sync, float32 accumulators).
//
// A request's portion is cut into chunks of 64 tokens from its first token on.  With S the state [N, P] that
// enters a chunk of n tokens, d_j the step sizes, L_i = -rate sum_{j <= i} d_j and i, j token indices in the chunk:
//
//     y_i   = e^(L_i) S^T C_i  +  sum_{j <= i} e^(L_i - L_j) d_j (C_i . B_j) x_j  +  skip x_i
//     S_out = e^(L_last) S     +  sum_j e^(L_last - L_j) d_j B_j x_j^T
//
// (all exponents are at most 0).  Three launches:
//
//   1. local sums   a block per (chunk, head, 64 value columns): sum_j e^(L_last - L_j) d_j B_j x_j^T, float32
//                   into a work buffer [chunks, H, N, P], and L_last;
//   2. scan         a thread per state element (or four) of a (request, head): walks the request's chunks in
//                   order, leaves in the work buffer the state that ENTERS each chunk and the final state in
//                   the request's slot;
//   3. outputs      a block per (chunk, head, 64 value columns): the formula for y_i.
//
// x, B and C are bfloat16 as the convolution left them, so they are exact operands.  What is float32 -- the
// weighted x of launch 1, the weighted scores and the entering state of launch 3 -- is staged as two bfloat16
// numbers, hi = bf16(a) and lo = bf16(a - hi), two MMAs a product (an error of about 2^-17 of the product's terms).
// Step sizes, their sums, exponentials and the state are float32.
#include "mma_util.cuh"
#include "state_space.cuh"

using namespace slb_mma;

#define SC_CHUNK 64
#define SC_THREADS 256
#define SC_PAD 8                   // bf16 elements added to every shared row (ldmatrix without bank conflicts)
#define SC_MAX_N 256
#define SC_EV 64                   // value columns a block
#define SC_LDX (SC_EV + SC_PAD)
#define SC_SCAN_BATCH 16

struct StateSpaceChunkArgs {
    StateSpaceArgs a;
    const int* tile_seq; const int* tile_row0; int num_tiles;
    float* work;                   // [num_tiles][H][N][P]
    float* total;                  // [num_tiles][H]: L_last
};

// the chunk's first token and its number of tokens
__device__ __forceinline__ bool sc_tile(const StateSpaceChunkArgs& c, int tile, int& t0, int& n, int& s) {
    s = c.tile_seq[tile];
    const int q0 = c.a.cu_q[s], row0 = c.tile_row0[tile];
    n = min(SC_CHUNK, c.a.cu_q[s + 1] - q0 - row0);
    t0 = q0 + row0;
    return n > 0;
}

// step sizes and their running sums times -rate (one warp, two tokens a lane; tokens from n on: 0 and L_last)
__device__ __forceinline__ void sc_steps(const StateSpaceArgs& a, int h, int t0, int n, float* d, float* L) {
    const int lane = threadIdx.x;
    const float bias = a.dt_bias[h], rate = a.rate[h];
    float d0 = 0.f, d1 = 0.f;
    if (2 * lane < n) d0 = ss_step(a.dt[(size_t)(t0 + 2 * lane) * a.ld_dt + h] + bias);
    if (2 * lane + 1 < n) d1 = ss_step(a.dt[(size_t)(t0 + 2 * lane + 1) * a.ld_dt + h] + bias);
    float sum = d0 + d1;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const float up = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += up;
    }
    const float before = sum - (d0 + d1);
    d[2 * lane] = d0;
    d[2 * lane + 1] = d1;
    L[2 * lane] = -rate * (before + d0);
    L[2 * lane + 1] = -rate * sum;
}

__device__ __forceinline__ void sc_zero(void* p, int bytes) {          // bytes a multiple of 16, p 16-byte aligned
    uint4* q = reinterpret_cast<uint4*>(p);
    for (int i = threadIdx.x; i < bytes / 16; i += SC_THREADS) q[i] = make_uint4(0, 0, 0, 0);
}

// `width` neighbouring elements of n rows, as they are
__device__ __forceinline__ void sc_stage(bf16* dst, int ldd, const bf16* src, int lds, int n, int width, bool wide) {
    if (wide) {
        const int wv = width >> 3;
        for (int idx = threadIdx.x; idx < n * wv; idx += SC_THREADS) {
            const int j = idx / wv, c = (idx - j * wv) << 3;
            *reinterpret_cast<uint4*>(dst + j * ldd + c) = *reinterpret_cast<const uint4*>(src + (size_t)j * lds + c);
        }
        return;
    }
    for (int idx = threadIdx.x; idx < n * width; idx += SC_THREADS) {
        const int j = idx / width, c = idx - j * width;
        dst[j * ldd + c] = src[(size_t)j * lds + c];
    }
}

// eight float32 numbers as hi and lo, `lo_off` elements apart
__device__ __forceinline__ void sc_put8(bf16* hi, int lo_off, int idx, const float (&x)[8]) {
    unsigned h[4], l[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        h[e] = pack_bf16(x[2 * e], x[2 * e + 1]);
        const __nv_bfloat162 hv = *reinterpret_cast<const __nv_bfloat162*>(&h[e]);
        l[e] = pack_bf16(x[2 * e] - __low2float(hv), x[2 * e + 1] - __high2float(hv));
    }
    *reinterpret_cast<uint4*>(hi + idx) = make_uint4(h[0], h[1], h[2], h[3]);
    *reinterpret_cast<uint4*>(hi + lo_off + idx) = make_uint4(l[0], l[1], l[2], l[3]);
}
__device__ __forceinline__ void sc_put(bf16* hi, int lo_off, int idx, float x) {
    const bf16 h = __float2bfloat16(x);
    hi[idx] = h;
    hi[lo_off + idx] = __float2bfloat16(x - __bfloat162float(h));
}

// rows of u whose pieces of 8 elements are whole 16-byte pieces
__device__ __forceinline__ bool sc_wide(const StateSpaceArgs& a) {
    return ((a.ld | a.x_off | a.b_off | a.c_off | a.P | a.N) & 7) == 0 && ((size_t)a.u & 15) == 0;
}

// ------------------------------------------------------------------ 1. local sums of a chunk
__global__ void __launch_bounds__(SC_THREADS) state_chunk_local_kernel(const StateSpaceChunkArgs c) {
    extern __shared__ __align__(16) unsigned char sc_smem[];
    __shared__ float d[SC_CHUNK], L[SC_CHUNK];
    pdl_wait();
    pdl_launch_dependents();
    const StateSpaceArgs& a = c.a;
    const int tile = blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * SC_EV;
    int t0, n, s;
    if (!sc_tile(c, tile, t0, n, s)) return;
    const int N = a.N, P = a.P, Np = (N + 15) & ~15, ldn = Np + SC_PAD;
    const int width = min(SC_EV, P - e0), grp = h / (a.H / a.G);
    const int x_elems = SC_CHUNK * SC_LDX;
    bf16* bs = reinterpret_cast<bf16*>(sc_smem);           // [64][ldn]
    bf16* xs = bs + SC_CHUNK * ldn;                        // [hi, lo][64][SC_LDX]
    if (n < SC_CHUNK || N < Np || width < SC_EV) {         // (a full tile is written whole)
        sc_zero(bs, (SC_CHUNK * ldn + 2 * x_elems) * (int)sizeof(bf16));
    }
    if (threadIdx.x < 32) sc_steps(a, h, t0, n, d, L);
    __syncthreads();
    const bf16* u = reinterpret_cast<const bf16*>(a.u) + (size_t)t0 * a.ld;
    const bool wide = sc_wide(a);
    const float last = L[SC_CHUNK - 1];
    if (threadIdx.x == 0 && e0 == 0) c.total[(size_t)tile * a.H + h] = last;
    sc_stage(bs, ldn, u + a.b_off + grp * N, a.ld, n, N, wide);
    const bf16* x = u + a.x_off + h * P + e0;
    if (wide) {
        const int wv = width >> 3;
        for (int idx = threadIdx.x; idx < n * wv; idx += SC_THREADS) {
            const int j = idx / wv, col = (idx - j * wv) << 3;
            const uint4 raw = *reinterpret_cast<const uint4*>(x + (size_t)j * a.ld + col);
            const unsigned w[4] = {raw.x, raw.y, raw.z, raw.w};
            const float f = d[j] * expf(last - L[j]);
            float v[8];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float2 p = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w[e]));
                v[2 * e] = p.x * f;
                v[2 * e + 1] = p.y * f;
            }
            sc_put8(xs, x_elems, j * SC_LDX + col, v);
        }
    } else {
        for (int idx = threadIdx.x; idx < n * width; idx += SC_THREADS) {
            const int j = idx / width, col = idx - j * width;
            sc_put(xs, x_elems, j * SC_LDX + col, to_float(x[(size_t)j * a.ld + col]) * d[j] * expf(last - L[j]));
        }
    }
    __syncthreads();

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int ksteps = (n + 15) >> 4;
    float* dst = c.work + ((size_t)tile * a.H + h) * (size_t)N * P;
    const bool pairs = !(P & 1);
    for (int unit = warp; unit < Np / 8; unit += SC_THREADS / 32) {       // 16 state rows x 32 value columns
        const int mt = unit >> 1, half = unit & 1;
        if (half * 32 >= width) continue;
        float acc[4][4];
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) acc[nt][0] = acc[nt][1] = acc[nt][2] = acc[nt][3] = 0.f;
        for (int kk = 0; kk < ksteps; ++kk) {
            // A[m = n][k = token] from rows stored [token][n]
            unsigned af[4];
            ldmatrix_x4_trans(af, bs + (kk * 16 + (lane & 7) + ((lane >> 4) & 1) * 8) * ldn + mt * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
            for (int np = 0; np < 2; ++np) {
                // B[k = token][n = e] from rows stored [token][e]
                const int b_at = (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * SC_LDX + half * 32 + np * 16 +
                                 ((lane >> 4) & 1) * 8;
                unsigned bh[4], bl[4];
                ldmatrix_x4_trans(bh, xs + b_at);
                ldmatrix_x4_trans(bl, xs + x_elems + b_at);
                mma_bf16(acc[2 * np], af, bl[0], bl[1]);
                mma_bf16(acc[2 * np], af, bh[0], bh[1]);
                mma_bf16(acc[2 * np + 1], af, bl[2], bl[3]);
                mma_bf16(acc[2 * np + 1], af, bh[2], bh[3]);
            }
        }
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
            const int e = e0 + half * 32 + nt * 8 + 2 * t;
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                const int row = mt * 16 + g + r * 8;
                if (row >= N) continue;
                float* o = dst + (size_t)row * P + e;
                if (pairs && e + 1 < P) {
                    *reinterpret_cast<float2*>(o) = make_float2(acc[nt][2 * r], acc[nt][2 * r + 1]);
                } else {
                    if (e < P) o[0] = acc[nt][2 * r];
                    if (e + 1 < P) o[1] = acc[nt][2 * r + 1];
                }
            }
        }
    }
}

// ------------------------------------------------------------------ 2. the states that enter the chunks
// A request's chunks are neighbours in the tile list, in order; the first one is found by a walk over the list.
template <int V>
__global__ void __launch_bounds__(256) state_chunk_scan_kernel(const StateSpaceChunkArgs c) {
    pdl_wait();
    pdl_launch_dependents();
    const StateSpaceArgs& a = c.a;
    const int s = blockIdx.x, h = blockIdx.y;
    const int qlen = a.cu_q[s + 1] - a.cu_q[s];
    if (qlen <= 0) return;
    const int slot = a.state_slots[s];
    if (slot < 0 || slot >= a.num_slots) return;
    const int elems = a.N * a.P;
    const int idx = (blockIdx.z * blockDim.x + threadIdx.x) * V;
    if (idx >= elems) return;
    int first = 0;
    while (first < c.num_tiles && c.tile_seq[first] != s) ++first;
    const int count = (qlen + SC_CHUNK - 1) / SC_CHUNK;
    if (first + count > c.num_tiles) return;
    float* sp = a.state + (size_t)slot * (size_t)a.state_stride + (size_t)h * elems + idx;
    float* wp = c.work + ((size_t)first * a.H + h) * (size_t)elems + idx;
    const float* lp = c.total + (size_t)first * a.H + h;
    const size_t step = (size_t)a.H * elems;
    float S[V];
    auto load = [](const float* p, float (&v)[V]) {
        if constexpr (V == 4) {
            const float4 x = *reinterpret_cast<const float4*>(p);
            v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
        } else {
            v[0] = p[0];
        }
    };
    auto store = [](float* p, const float (&v)[V]) {
        if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
        else p[0] = v[0];
    };
    load(sp, S);
    // (the loads of a batch do not wait for one another: one memory latency a batch, not a chunk)
    for (int k0 = 0; k0 < count; k0 += SC_SCAN_BATCH) {
        float add[SC_SCAN_BATCH][V], g[SC_SCAN_BATCH];
#pragma unroll
        for (int b = 0; b < SC_SCAN_BATCH; ++b) {
            const bool in = k0 + b < count;
            if (in) load(wp + b * step, add[b]);
            g[b] = in ? lp[(size_t)(k0 + b) * a.H] : 0.f;
        }
#pragma unroll
        for (int b = 0; b < SC_SCAN_BATCH; ++b) {
            if (k0 + b < count) {
                const float f = decay_exp(g[b]);
                store(wp + b * step, S);
#pragma unroll
                for (int v = 0; v < V; ++v) S[v] = fmaf(f, S[v], add[b][v]);
            }
        }
        wp += SC_SCAN_BATCH * step;
    }
    store(sp, S);
}

// ------------------------------------------------------------------ 3. the chunk's outputs
// Eight warps: 16 tokens and 32 of the value columns each (the scores of 16 tokens are formed by the two warps
// that share them).  The weighted scores stay in registers: the accumulator of C . B^T of 16 tokens x 16 tokens
// has the layout of the A operand of the product with x.  The entering state takes the place of B once the
// scores are formed.
__global__ void __launch_bounds__(SC_THREADS, 2) state_chunk_out_kernel(const StateSpaceChunkArgs c) {
    extern __shared__ __align__(16) unsigned char sc_smem[];
    __shared__ float d[SC_CHUNK], L[SC_CHUNK];
    pdl_wait();
    pdl_launch_dependents();
    const StateSpaceArgs& a = c.a;
    const int tile = blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * SC_EV;
    int t0, n, s;
    if (!sc_tile(c, tile, t0, n, s)) return;
    const int slot = a.state_slots[s];
    if (slot < 0 || slot >= a.num_slots) return;
    const int N = a.N, P = a.P, Np = (N + 15) & ~15, ldn = Np + SC_PAD;
    const int width = min(SC_EV, P - e0), grp = h / (a.H / a.G);
    const int n_elems = SC_CHUNK * ldn, s_elems = Np * SC_LDX;
    const int bs_elems = max(n_elems, 2 * s_elems);
    bf16* cs = reinterpret_cast<bf16*>(sc_smem);           // [64][ldn]
    bf16* xs = cs + n_elems;                               // [64][SC_LDX]
    bf16* bs = xs + SC_CHUNK * SC_LDX;                     // [64][ldn], later [hi, lo][Np][SC_LDX]
    if (n < SC_CHUNK || N < Np || width < SC_EV)
        sc_zero(cs, (n_elems + SC_CHUNK * SC_LDX + n_elems) * (int)sizeof(bf16));
    if (threadIdx.x < 32) sc_steps(a, h, t0, n, d, L);
    __syncthreads();
    const bf16* u = reinterpret_cast<const bf16*>(a.u) + (size_t)t0 * a.ld;
    const bool wide = sc_wide(a);
    sc_stage(cs, ldn, u + a.c_off + grp * N, a.ld, n, N, wide);
    sc_stage(bs, ldn, u + a.b_off + grp * N, a.ld, n, N, wide);
    sc_stage(xs, SC_LDX, u + a.x_off + h * P + e0, a.ld, n, width, wide);
    __syncthreads();

    const int warp = (threadIdx.x >> 5) & 3, wc = threadIdx.x >> 7;     // token group, half of the columns
    const int lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const bool live = warp * 16 < n && wc * 32 < width;
    const int a_row = (warp * 16 + (lane & 15)) * ldn + ((lane >> 4) & 1) * 8;   // A[m = token][k = n], + kk * 16
    const int i0 = warp * 16 + g;                           // this lane's two tokens: i0, i0 + 8

    float p[8][4];
#pragma unroll
    for (int nt = 0; nt < 8; ++nt) p[nt][0] = p[nt][1] = p[nt][2] = p[nt][3] = 0.f;
    if (live) {
        for (int kk = 0; kk < Np / 16; ++kk) {
            unsigned af[4];
            ldmatrix_x4(af, cs + a_row + kk * 16);
#pragma unroll
            for (int np = 0; np < 4; ++np) {
                if (np <= warp) {
                    // B[k = n][n = token] from rows stored [token][n]
                    unsigned bf[4];
                    ldmatrix_x4(bf, bs + (np * 16 + (lane & 7) + ((lane >> 4) & 1) * 8) * ldn + kk * 16 + ((lane >> 3) & 1) * 8);
                    mma_bf16(p[2 * np], af, bf[0], bf[1]);
                    mma_bf16(p[2 * np + 1], af, bf[2], bf[3]);
                }
            }
        }
        const float L0 = L[i0], L1 = L[i0 + 8];
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) {
            if (nt <= 2 * warp + 1) {
#pragma unroll
                for (int r = 0; r < 4; ++r) {
                    const int i = i0 + 8 * (r >> 1), j = nt * 8 + 2 * t + (r & 1);
                    p[nt][r] = (j <= i && i < n) ? p[nt][r] * (d[j] * expf((r >> 1 ? L1 : L0) - L[j])) : 0.f;
                }
            }
        }
    }
    __syncthreads();                                        // every warp is done with B

    // the entering state's tile [n][e] over it (padding rows and columns zero)
    {
        const float* src = c.work + ((size_t)tile * a.H + h) * (size_t)N * P + e0;
        if (N < Np || width < SC_EV) {
            sc_zero(bs, 2 * s_elems * (int)sizeof(bf16));
            __syncthreads();
        }
        if ((P & 7) == 0) {
            const int wv = width >> 3;
#pragma unroll 4
            for (int idx = threadIdx.x; idx < N * wv; idx += SC_THREADS) {
                const int row = idx / wv, col = (idx - row * wv) << 3;
                const float4 u0 = *reinterpret_cast<const float4*>(src + (size_t)row * P + col);
                const float4 u1 = *reinterpret_cast<const float4*>(src + (size_t)row * P + col + 4);
                const float v[8] = {u0.x, u0.y, u0.z, u0.w, u1.x, u1.y, u1.z, u1.w};
                sc_put8(bs, s_elems, row * SC_LDX + col, v);
            }
        } else {
            for (int idx = threadIdx.x; idx < N * width; idx += SC_THREADS) {
                const int row = idx / width, col = idx - row * width;
                sc_put(bs, s_elems, row * SC_LDX + col, src[(size_t)row * P + col]);
            }
        }
    }
    __syncthreads();
    if (!live) return;                                      // (no barrier follows)

    float acc[4][4];
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) acc[nt][0] = acc[nt][1] = acc[nt][2] = acc[nt][3] = 0.f;
    for (int kk = 0; kk < Np / 16; ++kk) {
        unsigned af[4];
        ldmatrix_x4(af, cs + a_row + kk * 16);
#pragma unroll
        for (int np = 0; np < 2; ++np) {
            // B[k = n][n = e] from rows stored [n][e]
            const int b_at = (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * SC_LDX + (wc * 2 + np) * 16 + ((lane >> 4) & 1) * 8;
            unsigned bh[4], bl[4];
            ldmatrix_x4_trans(bh, bs + b_at);
            ldmatrix_x4_trans(bl, bs + s_elems + b_at);
            mma_bf16(acc[2 * np], af, bl[0], bl[1]);
            mma_bf16(acc[2 * np], af, bh[0], bh[1]);
            mma_bf16(acc[2 * np + 1], af, bl[2], bl[3]);
            mma_bf16(acc[2 * np + 1], af, bh[2], bh[3]);
        }
    }
    {
        const float f0 = expf(L[i0]), f1 = expf(L[i0 + 8]);
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
            acc[nt][0] *= f0; acc[nt][1] *= f0;
            acc[nt][2] *= f1; acc[nt][3] *= f1;
        }
    }
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
        if (kk <= warp) {
            unsigned ah[4], al[4];
#pragma unroll
            for (int r = 0; r < 4; ++r) {
                const float x0 = p[2 * kk + (r >> 1)][2 * (r & 1)], x1 = p[2 * kk + (r >> 1)][2 * (r & 1) + 1];
                ah[r] = pack_bf16(x0, x1);
                const __nv_bfloat162 hv = *reinterpret_cast<const __nv_bfloat162*>(&ah[r]);
                al[r] = pack_bf16(x0 - __low2float(hv), x1 - __high2float(hv));
            }
#pragma unroll
            for (int np = 0; np < 2; ++np) {
                // B[k = token][n = e] from rows stored [token][e]
                unsigned bf[4];
                ldmatrix_x4_trans(bf, xs + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * SC_LDX + (wc * 2 + np) * 16 +
                                          ((lane >> 4) & 1) * 8);
                mma_bf16(acc[2 * np], al, bf[0], bf[1]);
                mma_bf16(acc[2 * np], ah, bf[0], bf[1]);
                mma_bf16(acc[2 * np + 1], al, bf[2], bf[3]);
                mma_bf16(acc[2 * np + 1], ah, bf[2], bf[3]);
            }
        }
    }
    const float skip = a.skip[h];
    const bool pairs = !((P | a.ldo) & 1);
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) {
        const int ec = (wc * 4 + nt) * 8 + 2 * t, e = e0 + ec;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int i = i0 + half * 8;
            if (i >= n) continue;
            const bf16* xr = xs + i * SC_LDX + ec;
            const float y0 = fmaf(skip, to_float(xr[0]), acc[nt][2 * half]);
            const float y1 = fmaf(skip, to_float(xr[1]), acc[nt][2 * half + 1]);
            float* o = a.out + (size_t)(t0 + i) * a.ldo + (size_t)h * P + e;
            if (pairs && e + 1 < P) {
                *reinterpret_cast<float2*>(o) = make_float2(y0, y1);
            } else {
                if (e < P) o[0] = y0;
                if (e + 1 < P) o[1] = y1;
            }
        }
    }
}

static size_t sc_local_smem(int N) {
    const int Np = (N + 15) & ~15;
    return ((size_t)SC_CHUNK * (Np + SC_PAD) + 2 * SC_CHUNK * SC_LDX) * sizeof(bf16);
}
static size_t sc_out_smem(int N) {
    const int Np = (N + 15) & ~15;
    const size_t rows = (size_t)SC_CHUNK * (Np + SC_PAD), st = (size_t)2 * Np * SC_LDX;
    return (rows + SC_CHUNK * SC_LDX + (rows > st ? rows : st)) * sizeof(bf16);
}

extern "C" {
int slb_state_space_chunk_tokens() { return SC_CHUNK; }
// u bfloat16; the tile list cuts every request's tokens of the step into chunks of slb_state_space_chunk_tokens()
// (request, first row), a request's in order.
int slb_state_space_chunk_bf16(const StateSpaceChunkArgs* c, int num_seqs, cudaStream_t st) {
    const StateSpaceArgs& a = c->a;
    if (num_seqs <= 0 || c->num_tiles <= 0) return 0;
    if (a.H <= 0 || a.P <= 0 || a.N <= 0 || a.G <= 0 || a.H % a.G != 0 || a.num_slots <= 0 ||
        a.state_stride < (long long)a.H * a.N * a.P || a.ldo < a.H * a.P || a.ld_dt < a.H || c->work == nullptr ||
        c->total == nullptr || c->tile_seq == nullptr || c->tile_row0 == nullptr ||
        (((uintptr_t)c->work | (uintptr_t)a.out) & 15))
        return SLB_ERR_BAD_ARG;
    if (a.N > SC_MAX_N || a.H > 65535 || a.P > 65535) return SLB_ERR_TOO_LARGE;
    static unsigned long long done_local = 0, done_out = 0;
    int rc = slb_configure(&done_local, state_chunk_local_kernel, sc_local_smem(SC_MAX_N));
    if (rc != 0) return rc;
    rc = slb_configure(&done_out, state_chunk_out_kernel, sc_out_smem(SC_MAX_N));
    if (rc != 0) return rc;
    const dim3 grid(c->num_tiles, a.H, (a.P + SC_EV - 1) / SC_EV);
    rc = slb_launch(state_chunk_local_kernel, grid, dim3(SC_THREADS), sc_local_smem(a.N), st, *c);
    if (rc != 0) return rc;
    const int elems = a.N * a.P;
    if (elems % 4 == 0 && a.state_stride % 4 == 0 && ((uintptr_t)a.state & 15) == 0)
        rc = slb_launch(state_chunk_scan_kernel<4>, dim3(num_seqs, a.H, (elems / 4 + 255) / 256), dim3(256), 0, st, *c);
    else
        rc = slb_launch(state_chunk_scan_kernel<1>, dim3(num_seqs, a.H, (elems + 255) / 256), dim3(256), 0, st, *c);
    if (rc != 0) return rc;
    return slb_launch(state_chunk_out_kernel, grid, dim3(SC_THREADS), sc_out_smem(a.N), st, *c);
}
}
