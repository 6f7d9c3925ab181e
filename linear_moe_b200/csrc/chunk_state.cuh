// A recurrent state in registers and the tiles that go into it, shared by the chunked recurrences (retention_tc.cu, ssd_tc.cu): 256 threads
// hold an fp32 state of up to 128 x 128 as mma.sync accumulators and add 64 tokens' keys times values at a time.
#pragma once
#include "mma_utils.cuh"

namespace lmoe {
namespace chk {

constexpr int CH = 64, NT = 256, PLD = CH + 8;               // tokens of a chunk, threads, row stride of a chunk's scores

template <int DK, int DV> struct Shape {
    static constexpr int LDK = DK + 8, LDV = DV + 8;         // row strides of the tiles
    static constexpr int RB = DK / 16, S_NT = DV / 8 / (8 / RB);         // row blocks of the state, its n-tiles per warp
    static constexpr int O_NT = DV / 16;                     // n-tiles of a warp's 16 x DV / 2 outputs
    static constexpr int KV = CH * LDK * 2 + CH * LDV * 2;   // bytes of a stage of keys and values
};

// [CH rows x cols] -> shared memory [CH][ld], columns up to D; rows from `valid` on and columns from `cols` on are zero
template <int D, int LD>
__device__ __forceinline__ void load_rows(bf16* smem, const bf16* g, long long pitch, int valid, int cols) {
    for (int i = threadIdx.x; i < CH * (D / 8); i += NT) {
        const int r = i / (D / 8), c = i % (D / 8) * 8;
        const bool ok = r < valid && c < cols;
        cp_async16(smem + r * LD + c, ok ? g + r * pitch + c : g, ok);
    }
}

template <int DK, int DV>
struct State {
    using C = Shape<DK, DV>;
    float s[C::S_NT][4];
    int m0, n0;                          // first row and column of this warp's part

    __device__ __forceinline__ State() {
        const int w = threadIdx.x >> 5;
        m0 = 16 * (w % C::RB), n0 = w / C::RB * (C::S_NT * 8);
    }
    __device__ __forceinline__ void load(const float* p, int dk, int dv) {           // null: zero
        const int l = threadIdx.x & 31, r = m0 + (l >> 2), c = n0 + (l & 3) * 2;
#pragma unroll
        for (int t = 0; t < C::S_NT; ++t)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const bool ok = p != nullptr && r + 8 * e < dk && c + 8 * t < dv;
                const float2 x = ok ? *reinterpret_cast<const float2*>(p + (long long)(r + 8 * e) * dv + c + 8 * t) : make_float2(0.f, 0.f);
                s[t][2 * e] = x.x, s[t][2 * e + 1] = x.y;
            }
    }
    __device__ __forceinline__ void store(float* p, int dk, int dv) const {
        const int l = threadIdx.x & 31, r = m0 + (l >> 2), c = n0 + (l & 3) * 2;
#pragma unroll
        for (int t = 0; t < C::S_NT; ++t)
#pragma unroll
            for (int e = 0; e < 2; ++e)
                if (r + 8 * e < dk && c + 8 * t < dv)
                    *reinterpret_cast<float2*>(p + (long long)(r + 8 * e) * dv + c + 8 * t) = make_float2(s[t][2 * e], s[t][2 * e + 1]);
    }
    // state <- whole * state + (factor(j) K_j)^T V_j over the chunk's tokens j (rows of tokens that are not there are zero)
    template <typename F>
    __device__ __forceinline__ void advance(const bf16* K, const bf16* V, float whole, F factor) {
        const int l = threadIdx.x & 31;
#pragma unroll
        for (int t = 0; t < C::S_NT; ++t)
#pragma unroll
            for (int e = 0; e < 4; ++e) s[t][e] *= whole;
#pragma unroll
        for (int k0 = 0; k0 < CH; k0 += 16) {
            uint32_t a[4];
            load_a_t(a, K, C::LDK, m0, k0);
#pragma unroll
            for (int e = 0; e < 4; ++e) {                    // registers 0, 1: tokens 2q, 2q + 1; registers 2, 3: eight later
                const int j = k0 + 8 * (e >> 1) + 2 * (l & 3);
                const float2 f = __bfloat1622float2(*reinterpret_cast<__nv_bfloat162*>(&a[e]));
                __nv_bfloat162 r = __floats2bfloat162_rn(f.x * factor(j), f.y * factor(j + 1));
                a[e] = *reinterpret_cast<uint32_t*>(&r);
            }
#pragma unroll
            for (int t = 0; t < C::S_NT; t += 2) {
                uint32_t b[4];
                load_b2_t(b, V, C::LDV, n0 + t * 8, k0);
                mma16816(s[t], a, b[0], b[1]);
                mma16816(s[t + 1], a, b[2], b[3]);
            }
        }
    }
};

}  // namespace chk
}  // namespace lmoe
