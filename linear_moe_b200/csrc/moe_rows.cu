// Mixture of experts over packed rows, for serving.  Scores are the sigmoid of the router logits or their softmax over all experts; the
// `top` largest are a token's experts, and its weights as they are or divided by their sum, times a factor.  Two kinds of experts:
//     squared ReLU   W_down relu(W_up (w h))^2 = W_down (w relu(W_up h))^2, because a weight is positive
//     gated          w W_down (silu(W_gate h) * (W_up h)) = W_down (w silu(W_gate h) * (W_up h))
// so the weight is applied in fp32 where the activation is formed and the rows themselves are never scaled.
//   route_rows_kernel     router logits -> experts and weights of every token (and the number of pairs per expert)
//   place_offsets_kernel  pairs per expert -> padded segments of the expert-sorted rows
//   place_rows_kernel     every (token, expert) pair gets a row of its expert's segment; its input row and weight go there
//   moe_rows_kernel       per-expert products over the sorted rows, any size, bf16 or fp32, fp32 arithmetic (the bf16 products of a
//                         prompt run on gemm_grouped.cu with the same activation in its epilogue)
//   moe_glu_kernel        the gated activation of the sorted rows
//   moe_step_kernel       the same products for few tokens (bf16): no sorting, every CTA finds its expert's pairs itself and streams 16
//                         rows of that expert's matrix through mma.sync fragments (as gemm_skinny.cu)
// Compiled without fast-math.
#include "common.cuh"
#include "mma_utils.cuh"

namespace lmoe {
namespace mr {

// ------------------------------------------------------------------------------------------------------------------ routing
constexpr int RT = 128;

// one warp per token; counts (null: not wanted) must be zero
__global__ void __launch_bounds__(RT) route_rows_kernel(const float* __restrict__ logits, long long ldl, int n, int E, int top, int softmax, int normalise, float scale,
                                                        int* __restrict__ idx, float* __restrict__ weight, int* counts) {
    pdl_trigger();
    const int t = blockIdx.x * (RT / 32) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (t >= n) return;
    const float* z = logits + (long long)t * ldl;
    float last = INFINITY;                                   // the previous choice; sigmoid and softmax keep the order of the logits
    int last_e = -1;
    float zmax = 0.f, inv = 0.f, chosen = 0.f;               // softmax: largest logit, 1 / sum; sum of the chosen scores
    if (softmax) {
        zmax = -INFINITY;
        for (int e = lane; e < E; e += 32) zmax = fmaxf(zmax, z[e]);
        zmax = warp_max(zmax);
        for (int e = lane; e < E; e += 32) inv += expf(z[e] - zmax);
        inv = 1.f / warp_sum(inv);
    }
    for (int k = 0; k < top; ++k) {
        float best = -INFINITY;
        int be = E;
        for (int e = lane; e < E; e += 32) {
            const float v = z[e];
            const bool after = v < last || (v == last && e > last_e);      // not chosen yet (equal logits: by index)
            if (after && (v > best || be == E)) { best = v; be = e; }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, best, o);
            const int oe = __shfl_xor_sync(0xffffffffu, be, o);
            if (oe < E && (be == E || ov > best || (ov == best && oe < be))) { best = ov; be = oe; }
        }
        last = best;
        last_e = be;
        if (lane == 0) {
            const int e = min(be, E - 1);                    // (logits that are no numbers leave nothing to choose)
            idx[(long long)t * top + k] = e;
            const float s = be == E ? 0.f : softmax ? expf(best - zmax) * inv : 1.f / (1.f + expf(-best));
            weight[(long long)t * top + k] = normalise ? s : s * scale;
            chosen += s;
            if (counts != nullptr) atomicAdd(counts + e, 1);
        }
    }
    if (normalise && lane == 0)
        for (int k = 0; k < top; ++k) weight[(long long)t * top + k] = weight[(long long)t * top + k] / (chosen + 1e-20f) * scale;
}

__global__ void place_offsets_kernel(const int* __restrict__ counts, int* __restrict__ offs, int E, int align) {
    __shared__ int part[1024];
    int base = 0;                                            // padded rows of the experts before this pass
    for (int e0 = 0; e0 < E; e0 += blockDim.x) {
        const int e = e0 + threadIdx.x;
        int v = e < E ? (counts[e] + align - 1) / align * align : 0;
        part[threadIdx.x] = v;
        __syncthreads();
        for (int o = 1; o < blockDim.x; o <<= 1) {
            const int add = threadIdx.x >= o ? part[threadIdx.x - o] : 0;
            __syncthreads();
            part[threadIdx.x] += add;
            __syncthreads();
        }
        if (e < E) offs[e + 1] = base + part[threadIdx.x];
        base += part[blockDim.x - 1];
        __syncthreads();
    }
    if (threadIdx.x == 0) offs[0] = 0;
}

// one warp per pair; cursor must be zero.  The order of an expert's rows is arbitrary, their results do not depend on it.
template <typename T>
__global__ void __launch_bounds__(RT) place_rows_kernel(const T* __restrict__ h, long long ldh, const int* __restrict__ idx,
                                                        const float* __restrict__ weight, const int* __restrict__ offs, int* cursor,
                                                        T* __restrict__ xs, long long ldxs, float* __restrict__ ws, int* __restrict__ dest,
                                                        int pairs, int top, int cols) {
    constexpr int W = Vec<T>::N;
    const int p = blockIdx.x * (RT / 32) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (p >= pairs) return;
    int row = 0;
    if (lane == 0) {
        const int e = idx[p];
        row = offs[e] + atomicAdd(cursor + e, 1);
        dest[p] = row;
        ws[row] = weight[p];
    }
    row = __shfl_sync(0xffffffffu, row, 0);
    const T* src = h + (long long)(p / top) * ldh;
    T* dst = xs + (long long)row * ldxs;
    for (int c = lane * W; c < cols; c += 32 * W) {
        Vec<T> v;
        v.load(src + c);
        v.store(dst + c);
    }
}

// ------------------------------------------------------------------------------------------------- products, any size and type
constexpr int GT = 64, GK = 16;

// C[row, :N] = X[row, :K] W[e][:N, :K]^T for the rows of expert e; row_scale: (scale * relu(.))^2.  grid (N tiles, row tiles)
template <typename T>
__global__ void __launch_bounds__(256) moe_rows_kernel(const T* __restrict__ X, long long ldx, const T* __restrict__ Wt, T* __restrict__ C,
                                                       long long ldc, const int* __restrict__ offs, const float* __restrict__ row_scale, int E,
                                                       int N, int K) {
    __shared__ float As[GK][GT + 4], Bs[GK][GT + 4];
    __shared__ int expert;
    const int row0 = blockIdx.y * GT, col0 = blockIdx.x * GT;
    if (row0 >= offs[E]) return;                             // segments are padded to GT rows: a tile has one expert
    for (int e = threadIdx.x; e < E; e += 256)
        if (offs[e] <= row0 && row0 < offs[e + 1]) expert = e;
    __syncthreads();
    const T* W = Wt + (long long)expert * N * K;
    const int ty = threadIdx.x / 16, tx = threadIdx.x % 16;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < K; k0 += GK) {
        __syncthreads();
        for (int i = threadIdx.x; i < GT * GK; i += 256) {
            const int r = i / GK, k = i % GK;
            As[k][r] = k0 + k < K ? to_f(X[(long long)(row0 + r) * ldx + k0 + k]) : 0.f;
            Bs[k][r] = k0 + k < K && col0 + r < N ? to_f(W[(long long)(col0 + r) * K + k0 + k]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < GK; ++k) {
            const float4 a = *reinterpret_cast<const float4*>(&As[k][4 * ty]), b = *reinterpret_cast<const float4*>(&Bs[k][4 * tx]);
            const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] += av[i] * bv[j];
        }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const long long r = row0 + 4 * ty + i;
        const float w = row_scale == nullptr ? 0.f : row_scale[r];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int c = col0 + 4 * tx + j;
            if (c < N) {
                const float a = row_scale == nullptr ? acc[i][j] : w * fmaxf(acc[i][j], 0.f);
                C[r * ldc + c] = from_f<T>(row_scale == nullptr ? a : a * a);
            }
        }
    }
}

// z [rows, ldz]: gate in columns 0 .. ff, up in ff .. 2 ff -> out[row] = row_scale[row] silu(gate) * up for the rows in use
template <typename T>
__global__ void __launch_bounds__(256) moe_glu_kernel(const T* __restrict__ z, long long ldz, T* __restrict__ out, long long ldo, const int* __restrict__ used,
                                                      const float* __restrict__ row_scale, int rows, int ff) {
    pdl_trigger();
    constexpr int W = Vec<T>::N;
    const int pieces = ff / W;
    const long long total = (long long)min(rows, *used) * pieces;
    for (long long i = blockIdx.x * 256LL + threadIdx.x; i < total; i += gridDim.x * 256LL) {
        const long long row = i / pieces;
        const int c = (int)(i - row * pieces) * W;
        const float w = row_scale[row];
        Vec<T> g, u;
        g.load(z + row * ldz + c);
        u.load(z + row * ldz + ff + c);
#pragma unroll
        for (int e = 0; e < W; ++e) {
            const float t = g.get(e);
            g.set(e, w * (sizeof(T) == 2 ? __fdividef(t, 1.f + __expf(-t)) : t / (1.f + expf(-t))) * u.get(e));
        }
        g.store(out + row * ldo + c);
    }
}

// --------------------------------------------------------------------------------------------------------------- few tokens
constexpr int SW = 8, MAX_PAIRS = 1024;

// One product for every pair p (token p / top, expert idx[p]); grid (N / 16 rounded up, E; GATED: N / 8).
//   RELU2  x row p / top of h,  y[p] = (weight[p] * relu(.))^2 in bf16
//   GATED  x row p / top of h,  y[p] = weight[p] * silu(.) * (.) in bf16 with the N gate rows in front of the N up rows of an expert's matrix
//   DOWN   x row p,             y[p] in fp32
enum Kind { DOWN, RELU2, GATED };
template <Kind KIND>
__global__ void __launch_bounds__(SW * 32) moe_step_kernel(const bf16* __restrict__ x, long long ldx, const bf16* __restrict__ Wt, void* y,
                                                           long long ldy, const int* __restrict__ idx, const float* __restrict__ weight,
                                                           int pairs, int top, int N, int K) {
    __shared__ float red[SW][2][32][4];
    __shared__ int list[MAX_PAIRS], count;
    const int w = threadIdx.x >> 5, l = threadIdx.x & 31, g = l >> 2, q = l & 3;
    constexpr bool UP = KIND != DOWN;
    constexpr int ROWS = KIND == GATED ? 8 : 16;             // outputs of a CTA: its fragments' lower rows are up rows of the same outputs
    const int e = blockIdx.y, r0 = blockIdx.x * ROWS;
    pdl_trigger();
    asm volatile("griddepcontrol.wait;" ::: "memory");
    if (w == 0) {                                            // this expert's pairs, in order
        int n = 0;
        for (int p0 = 0; p0 < pairs; p0 += 32) {
            const bool mine = p0 + l < pairs && idx[p0 + l] == e;
            const unsigned m = __ballot_sync(0xffffffffu, mine);
            if (mine) list[n + __popc(m & ((1u << l) - 1))] = p0 + l;
            n += __popc(m);
        }
        if (l == 0) count = n;
    }
    __syncthreads();
    const int n = count;
    if (n == 0) return;
    const bool lo_ok = r0 + g < N, hi_ok = KIND == GATED ? lo_ok : r0 + g + 8 < N;
    const long long M = KIND == GATED ? 2LL * N : N;         // rows of an expert's matrix
    const bf16* w_lo = Wt + (e * M + (lo_ok ? r0 + g : 0)) * K + q * 8;
    const bf16* w_hi = Wt + (e * M + (hi_ok ? r0 + g + (KIND == GATED ? N : 8) : 0)) * K + q * 8;
    const uint4 zero = make_uint4(0, 0, 0, 0);
    for (int n0 = 0; n0 < n; n0 += 16) {                     // 16 pairs at a time; another round reads the weights from L1 / L2
        const bf16* xr[2];
        bool on[2];
#pragma unroll
        for (int t = 0; t < 2; ++t) {
            on[t] = n0 + 8 * t + g < n;
            const int p = list[on[t] ? n0 + 8 * t + g : 0];
            xr[t] = x + (long long)(UP ? p / top : p) * ldx + q * 8;
        }
        const bool two = n0 + 8 < n;
        float acc[2][4];
#pragma unroll
        for (int t = 0; t < 2; ++t) acc[t][0] = acc[t][1] = acc[t][2] = acc[t][3] = 0.f;
#pragma unroll 8
        for (int k0 = w * 32; k0 < K; k0 += SW * 32) {
            const uint4 lo = lo_ok ? *reinterpret_cast<const uint4*>(w_lo + k0) : zero, hi = hi_ok ? *reinterpret_cast<const uint4*>(w_hi + k0) : zero;
            const uint32_t a1[4] = {lo.x, hi.x, lo.y, hi.y}, a2[4] = {lo.z, hi.z, lo.w, hi.w};
            const uint4 b = on[0] ? *reinterpret_cast<const uint4*>(xr[0] + k0) : zero;
            mma16816(acc[0], a1, b.x, b.y);
            mma16816(acc[0], a2, b.z, b.w);
            if (two) {
                const uint4 c = on[1] ? *reinterpret_cast<const uint4*>(xr[1] + k0) : zero;
                mma16816(acc[1], a1, c.x, c.y);
                mma16816(acc[1], a2, c.z, c.w);
            }
        }
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
            for (int i = 0; i < 4; ++i) red[w][t][l][i] = acc[t][i];
        __syncthreads();
        if (w < 2) {
#pragma unroll
            for (int i = 0; i < (KIND == GATED ? 2 : 4); ++i) {
                const int b = n0 + 8 * w + 2 * q + (i & 1), r = r0 + g + 8 * (i >> 1);
                if (b < n && r < N) {
                    float s = 0.f;
#pragma unroll
                    for (int k = 0; k < SW; ++k) s += red[k][w][l][i];
                    const int p = list[b];
                    if (KIND == GATED) {
                        float u = 0.f;
#pragma unroll
                        for (int k = 0; k < SW; ++k) u += red[k][w][l][i + 2];
                        ((bf16*)y)[(long long)p * ldy + r] = __float2bfloat16(weight[p] * (s / (1.f + expf(-s))) * u);
                    } else if (KIND == RELU2) {
                        s = weight[p] * fmaxf(s, 0.f);
                        ((bf16*)y)[(long long)p * ldy + r] = __float2bfloat16(s * s);
                    } else {
                        ((float*)y)[(long long)p * ldy + r] = s;
                    }
                }
            }
        }
        __syncthreads();
    }
}

template <Kind KIND>
static int launch_step(const bf16* x, long long ldx, const bf16* W, void* y, long long ldy, const int* idx, const float* weight, int pairs,
                       int top, int E, int N, int K, cudaStream_t st) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(KIND == GATED ? (N + 7) / 8 : (N + 15) / 16, E);
    cfg.blockDim = dim3(SW * 32);
    cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    return (int)cudaLaunchKernelEx(&cfg, moe_step_kernel<KIND>, x, ldx, W, y, ldy, idx, weight, pairs, top, N, K);
}

}  // namespace mr
}  // namespace lmoe

using namespace lmoe;

// logits [n, ldl] fp32 -> idx, weight [n, top] (largest first); softmax: scores over all experts instead of each one's sigmoid; normalise: weights
// over their sum; counts [E] zeros or null
LMOE_API int lmoe_route_rows(const float* logits, long long ldl, int n, int E, int top, int softmax, int normalise, float scale, int* idx, float* weight, int* counts, cudaStream_t st) {
    if (n <= 0 || E <= 0 || top <= 0 || top > E) return -1;
    mr::route_rows_kernel<<<(n + mr::RT / 32 - 1) / (mr::RT / 32), mr::RT, 0, st>>>(logits, ldl, n, E, top, softmax, normalise, scale,
                                                                                                idx, weight, counts);
    return (int)cudaGetLastError();
}

// offs [E + 1] (segments padded to `align` rows), then every pair's row: xs [offs[E], ldxs], ws, dest [n * top].  cursor [E] zeros.
LMOE_API int lmoe_place_rows(const void* h, long long ldh, const int* idx, const float* weight, const int* counts, int* offs, int* cursor,
                             void* xs, long long ldxs, float* ws, int* dest, int n, int top, int E, int align, int cols, int dt,
                             cudaStream_t st) {
    const int w = dt ? 8 : 4;
    if (n <= 0 || top <= 0 || E <= 0 || align <= 0 || cols <= 0 || cols % w || ldh % w || ldxs % w ||
        ((reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(xs)) & 15))
        return -1;
    const int threads = E <= 256 ? 256 : 1024;
    mr::place_offsets_kernel<<<1, threads, 0, st>>>(counts, offs, E, align);
    const int pairs = n * top, blocks = (pairs + mr::RT / 32 - 1) / (mr::RT / 32);
    if (dt) mr::place_rows_kernel<bf16><<<blocks, mr::RT, 0, st>>>((const bf16*)h, ldh, idx, weight, offs, cursor, (bf16*)xs, ldxs, ws, dest, pairs, top, cols);
    else mr::place_rows_kernel<float><<<blocks, mr::RT, 0, st>>>((const float*)h, ldh, idx, weight, offs, cursor, (float*)xs, ldxs, ws, dest, pairs, top, cols);
    return (int)cudaGetLastError();
}

// X [max_rows, ldx], W [E, N, K], C [max_rows, ldc]; offsets multiples of 64; row_scale [max_rows] or null
LMOE_API int lmoe_moe_rows(const void* X, long long ldx, const void* W, void* C, long long ldc, const int* offs, const float* row_scale,
                           int max_rows, int E, int N, int K, int dt, cudaStream_t st) {
    if (max_rows <= 0 || max_rows % mr::GT || E <= 0 || N <= 0 || K <= 0 || max_rows / mr::GT > 65535) return -1;
    const dim3 grid((N + mr::GT - 1) / mr::GT, max_rows / mr::GT);
    if (dt) mr::moe_rows_kernel<bf16><<<grid, 256, 0, st>>>((const bf16*)X, ldx, (const bf16*)W, (bf16*)C, ldc, offs, row_scale, E, N, K);
    else mr::moe_rows_kernel<float><<<grid, 256, 0, st>>>((const float*)X, ldx, (const float*)W, (float*)C, ldc, offs, row_scale, E, N, K);
    return (int)cudaGetLastError();
}

// z [rows, ldz] -> out [rows, ldo]; offs [E + 1]: the rows in use end at offs[E]
LMOE_API int lmoe_moe_glu(const void* z, long long ldz, void* out, long long ldo, const int* offs, const float* row_scale, int rows, int E, int ff, int dt,
                          cudaStream_t st) {
    const int w = dt ? 8 : 4;
    if (rows <= 0 || E <= 0 || ff <= 0 || ff % w || ldz % w || ldo % w || offs == nullptr || row_scale == nullptr ||
        ((reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(out)) & 15))
        return -1;
    const long long blocks = ((long long)rows * (ff / w) + 255) / 256;
    const unsigned grid = (unsigned)(blocks < 148 * 16 ? blocks : 148 * 16);
    if (dt) mr::moe_glu_kernel<bf16><<<grid, 256, 0, st>>>((const bf16*)z, ldz, (bf16*)out, ldo, offs + E, row_scale, rows, ff);
    else mr::moe_glu_kernel<float><<<grid, 256, 0, st>>>((const float*)z, ldz, (float*)out, ldo, offs + E, row_scale, rows, ff);
    return (int)cudaGetLastError();
}

// kind 1 (squared ReLU), 2 (gated): x [n, ldx] -> y [n * top, ldy] bf16;  0 (down): x [n * top, ldx] -> y [n * top, ldy] fp32.  K a multiple of 32, ldx of 8, at most 1024 pairs
LMOE_API int lmoe_moe_step(const bf16* x, long long ldx, const bf16* W, void* y, long long ldy, const int* idx, const float* weight, int n,
                           int top, int E, int N, int K, int kind, cudaStream_t st) {
    if (n <= 0 || top <= 0 || (long long)n * top > mr::MAX_PAIRS || E <= 0 || E > 65535 || N <= 0 || K <= 0 || K % 32 || ldx % 8 ||
        kind < 0 || kind > 2 ||
        ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(W)) & 15))
        return -1;
    return kind == 2   ? mr::launch_step<mr::GATED>(x, ldx, W, y, ldy, idx, weight, n * top, top, E, N, K, st)
           : kind == 1 ? mr::launch_step<mr::RELU2>(x, ldx, W, y, ldy, idx, weight, n * top, top, E, N, K, st)
                       : mr::launch_step<mr::DOWN>(x, ldx, W, y, ldy, idx, weight, n * top, top, E, N, K, st);
}
