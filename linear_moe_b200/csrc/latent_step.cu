// The per-head products around one-token latent attention (bf16).  With the cached latent row c, k = W_uk c and v = W_uv c of a
// head, the scores are q . (W_uk c) = (W_uk^T q) . c and the output is W_uv (sum of p c): a step never forms keys or values.
//   latent_absorb_kernel   q'[n, h] = W_uk[h]^T q[n, h]
//   latent_up_kernel       o[n, h] = sigmoid(gate) * W_uv[h] o'[n, h]
// Both stream a head's matrix once per 16 requests through mma.sync fragments loaded from global memory (as gemm_skinny.cu); the
// four warps of a CTA split the sum.  Launched with programmatic stream serialization: the weights are on their way before the
// kernel that produces the other operand has ended.
#include "attn_math.cuh"
#include "mma_utils.cuh"

namespace lmoe {
namespace lat {

constexpr int WARPS = 4, NB = 16;        // warps, requests per CTA
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ uint32_t word(const uint4& v, int i) { return i == 0 ? v.x : i == 1 ? v.y : i == 2 ? v.z : v.w; }

// W [H * dk, rank]; grid (rank / 64 rounded up, H, n / 16 rounded up)
__global__ void __launch_bounds__(WARPS * 32) latent_absorb_kernel(const bf16* __restrict__ qm, long long ldq, const bf16* __restrict__ W,
                                                                   bf16* __restrict__ out, long long ldo, int n, int dk, int rank) {
    __shared__ float red[WARPS][NB][64 + 1];
    const int w = threadIdx.x >> 5, l = threadIdx.x & 31, g = l >> 2, q = l & 3;
    const int h = blockIdx.y, r0 = blockIdx.x * 64, n0 = blockIdx.z * NB;
    const bf16* Wh = W + (long long)h * dk * rank;
    const bool on = r0 + g * 8 < rank;
    const uint4 zero = make_uint4(0, 0, 0, 0);
    auto load = [&](uint4 (&f)[4], int d0) {                  // rows of W whose k slots this lane owns, eight latent columns each
#pragma unroll
        for (int r = 0; r < 4; ++r)
            f[r] = on && d0 < dk ? *reinterpret_cast<const uint4*>(Wh + (long long)(d0 + 2 * q + (r & 1) + 8 * (r >> 1)) * rank + r0 + g * 8) : zero;
    };
    uint4 f[2][4];
    load(f[0], w * 16);
    load(f[1], (w + WARPS) * 16);
    pdl_trigger();
    asm volatile("griddepcontrol.wait;" ::: "memory");
    float o[2][4][4];
#pragma unroll
    for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int i = 0; i < 4; ++i) o[t][i][0] = o[t][i][1] = o[t][i][2] = o[t][i][3] = 0.f;
    for (int d0 = w * 16, i = 0; d0 < dk; d0 += WARPS * 16, ++i) {
        uint4 cur[4];
        if (i < 2) {
#pragma unroll
            for (int r = 0; r < 4; ++r) cur[r] = i == 0 ? f[0][r] : f[1][r];
        } else {
            load(cur, d0);
        }
#pragma unroll
        for (int t = 0; t < 2; ++t) {
            const int row = n0 + 8 * t + g;
            const bf16* p = qm + (long long)row * ldq + (long long)h * dk + d0 + 2 * q;
            const uint32_t b0 = row < n ? *reinterpret_cast<const uint32_t*>(p) : 0u, b1 = row < n ? *reinterpret_cast<const uint32_t*>(p + 8) : 0u;
#pragma unroll
            for (int e = 0; e < 4; ++e) {                     // rows g, g + 8 of the tile: columns 2e, 2e + 1 of this lane's eight
                const uint32_t w0 = word(cur[0], e), w1 = word(cur[1], e), w2 = word(cur[2], e), w3 = word(cur[3], e);
                const uint32_t a[4] = {__byte_perm(w0, w1, 0x5410), __byte_perm(w0, w1, 0x7632), __byte_perm(w2, w3, 0x5410),
                                       __byte_perm(w2, w3, 0x7632)};
                mma16816(o[t][e], a, b0, b1);
            }
        }
    }
#pragma unroll
    for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int c = g * 8 + 2 * e;
            red[w][8 * t + 2 * q][c] = o[t][e][0];
            red[w][8 * t + 2 * q + 1][c] = o[t][e][1];
            red[w][8 * t + 2 * q][c + 1] = o[t][e][2];
            red[w][8 * t + 2 * q + 1][c + 1] = o[t][e][3];
        }
    __syncthreads();
    for (int i = threadIdx.x; i < NB * 64; i += WARPS * 32) {
        const int b = i / 64, c = i % 64;
        if (n0 + b < n && r0 + c < rank) {
            float s = 0.f;
#pragma unroll
            for (int k = 0; k < WARPS; ++k) s += red[k][b][c];
            out[(long long)(n0 + b) * ldo + (long long)h * rank + r0 + c] = __float2bfloat16(s);
        }
    }
}

// W [H * dv, rank]; grid (dv / 16 rounded up, H, n / 16 rounded up)
__global__ void __launch_bounds__(WARPS * 32) latent_up_kernel(const bf16* __restrict__ x, long long ldx, const bf16* __restrict__ W,
                                                               const bf16* __restrict__ gate, long long ldg, bf16* __restrict__ out,
                                                               long long ldo, int n, int dv, int rank) {
    __shared__ float red[WARPS][2][32][4];
    const int w = threadIdx.x >> 5, l = threadIdx.x & 31, g = l >> 2, q = l & 3;
    const int h = blockIdx.y, v0 = blockIdx.x * 16, n0 = blockIdx.z * NB;
    const bool lo_ok = v0 + g < dv, hi_ok = v0 + g + 8 < dv;
    const bf16* w_lo = W + ((long long)h * dv + (lo_ok ? v0 + g : 0)) * rank + q * 8;
    const bf16* w_hi = W + ((long long)h * dv + (hi_ok ? v0 + g + 8 : 0)) * rank + q * 8;
    const uint4 zero = make_uint4(0, 0, 0, 0);
    constexpr int PF = 4;
    uint4 f_lo[PF], f_hi[PF];
#pragma unroll
    for (int i = 0; i < PF; ++i) {
        const int k0 = (w + i * WARPS) * 32;
        f_lo[i] = lo_ok && k0 < rank ? *reinterpret_cast<const uint4*>(w_lo + k0) : zero;
        f_hi[i] = hi_ok && k0 < rank ? *reinterpret_cast<const uint4*>(w_hi + k0) : zero;
    }
    pdl_trigger();
    asm volatile("griddepcontrol.wait;" ::: "memory");
    float acc[2][4];
#pragma unroll
    for (int t = 0; t < 2; ++t) acc[t][0] = acc[t][1] = acc[t][2] = acc[t][3] = 0.f;
    auto step = [&](const uint4& lo, const uint4& hi, int k0) {
        const uint32_t a1[4] = {lo.x, hi.x, lo.y, hi.y}, a2[4] = {lo.z, hi.z, lo.w, hi.w};
#pragma unroll
        for (int t = 0; t < 2; ++t) {
            const int row = n0 + 8 * t + g;
            const uint4 b = row < n ? *reinterpret_cast<const uint4*>(x + (long long)row * ldx + (long long)h * rank + q * 8 + k0) : zero;
            mma16816(acc[t], a1, b.x, b.y);
            mma16816(acc[t], a2, b.z, b.w);
        }
    };
#pragma unroll
    for (int i = 0; i < PF; ++i) {
        const int k0 = (w + i * WARPS) * 32;
        if (k0 < rank) step(f_lo[i], f_hi[i], k0);
    }
    for (int k0 = (w + PF * WARPS) * 32; k0 < rank; k0 += WARPS * 32)
        step(lo_ok ? *reinterpret_cast<const uint4*>(w_lo + k0) : zero, hi_ok ? *reinterpret_cast<const uint4*>(w_hi + k0) : zero, k0);
#pragma unroll
    for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) red[w][t][l][e] = acc[t][e];
    __syncthreads();
    if (w < 2) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int b = n0 + 8 * w + 2 * q + (e & 1), v = v0 + g + 8 * (e >> 1);
            if (b < n && v < dv) {
                float s = 0.f;
#pragma unroll
                for (int k = 0; k < WARPS; ++k) s += red[k][w][l][e];
                const float z = __bfloat162float(gate[(long long)b * ldg + (long long)h * dv + v]);
                out[(long long)b * ldo + (long long)h * dv + v] = __float2bfloat16(s * rcp(1.f + ex2(-LOG2E * z)));
            }
        }
    }
}

template <typename K, typename... A>
static int launch(K kern, dim3 grid, cudaStream_t st, A... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = dim3(WARPS * 32);
    cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    return (int)cudaLaunchKernelEx(&cfg, kern, args...);
}

static bool aligned(const void* a, const void* b, const void* c) {
    return ((reinterpret_cast<uintptr_t>(a) | reinterpret_cast<uintptr_t>(b) | reinterpret_cast<uintptr_t>(c)) & 15) == 0;
}

}  // namespace lat
}  // namespace lmoe

using namespace lmoe;

// q [n, ldq] (head by head dk columns), W [H * dk, rank], out [n, ldo] (head by head rank columns); dk a multiple of 16, rank of 32, ldq
// of 8, 16-byte aligned bases
LMOE_API int lmoe_latent_absorb(const bf16* q, long long ldq, const bf16* W, bf16* out, long long ldo, int n, int H, int dk, int rank,
                                cudaStream_t st) {
    if (n <= 0 || H <= 0 || dk <= 0 || rank <= 0 || dk % 16 || rank % 32 || ldq % 8 || !lat::aligned(q, W, out)) return -1;
    return lat::launch(lat::latent_absorb_kernel, dim3((rank + 63) / 64, H, (n + lat::NB - 1) / lat::NB), st, q, ldq, W, out, ldo, n, dk, rank);
}

// x [n, ldx] (head by head rank columns), W [H * dv, rank], gate and out [n, ld] (head by head dv columns)
LMOE_API int lmoe_latent_up(const bf16* x, long long ldx, const bf16* W, const bf16* gate, long long ldg, bf16* out, long long ldo, int n,
                            int H, int dv, int rank, cudaStream_t st) {
    if (n <= 0 || H <= 0 || dv <= 0 || rank <= 0 || rank % 32 || ldx % 8 || !lat::aligned(x, W, out)) return -1;
    return lat::launch(lat::latent_up_kernel, dim3((dv + 15) / 16, H, (n + lat::NB - 1) / lat::NB), st, x, ldx, W, gate, ldg, out, ldo, n, dv, rank);
}
