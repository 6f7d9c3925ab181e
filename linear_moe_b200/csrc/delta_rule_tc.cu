// The generalized delta rule over prompts for bf16 (definition and arguments: delta_rule.cu, delta_rule.cuh), head sizes up to 128: chunks of 64
// tokens on tensor-core fragments (mma.sync), the state in fp32.
//
// In a chunk let L_t be the sum of the log decays up to token t (per channel) and, row by row,
//     U_t = u e^{L_{t-1}},  B_t = a u e^{-L_t},  K_t = k e^{-L_t},  R_t = r e^{L_t}.
// A log decay is at least -DECAY, so these stay far inside the range of bf16, and every product of two of them that is used decays.  What the
// tokens read from the state along their keys, p_t = u_t^T S_{t-1}, obeys (I + tril(U B^T, -1)) P = U S + tril(U K^T, -1) V with the state S in
// front of the chunk.  With M the inverse on the left, G = M U and H = M tril(U K^T, -1) V (found by substitution in blocks of 16),
//     O  = Q S + N,     Q = R - tril(R B^T) G,    N = tril(R K^T) V - tril(R B^T) H
//     S' = e^{L} S - E S + D,     E = e^{L} B^T G,    D = e^{L} (K^T V - B^T H)              (e^{L} of the whole chunk, row by row)
//   delta_chunk_kernel   Q, N, E, D and e^{L} of every chunk, all in parallel
//   delta_pass_kernel    the states in front of the chunks, one request and head after the other's chunks, 32 columns of the state per CTA
//   delta_out_kernel     O of every chunk, norm and gate
#include "chunk_state.cuh"
#include "delta_rule.cuh"

namespace lmoe {
namespace dltc {
using namespace chk;
using namespace rt;
using dlt::Args;
using dlt::DECAY;
using dlt::UNIT_EPS;

// of a request, in `groups` behind the chunks' entries: slot, flags, first chunk, chunks
enum { Q_SLOT, Q_FLAGS, Q_FIRST, Q_CHUNKS };

// what a chunk of a head leaves, as laid out in `work`: [chunks, H] of each
template <int D> struct Work {
    float *N, *Dm, *decay;               // [CH, D], [D, D], [D]
    bf16 *Q, *E, *S;                     // [CH, D], [D, D], [D, D]
    __device__ __forceinline__ Work(void* work, long long all, long long i) {
        float* f = (float*)work;
        N = f + i * CH * D;
        f += all * CH * D;
        Dm = f + i * D * D;
        f += all * D * D;
        decay = f + i * D;
        f += all * D;
        bf16* b = (bf16*)f;
        Q = b + i * CH * D;
        b += all * CH * D;
        E = b + i * D * D;
        b += all * D * D;
        S = b + i * D * D;
    }
};

__device__ __forceinline__ float sigmoid(float x) { return 1.f / (1.f + __expf(-x)); }

template <int D> struct Cfg {
    static constexpr int LD = D + 8, SEGS = NT / D, SEG = CH / SEGS;     // segments of tokens a thread sums the log decays over
    static constexpr int TILE = CH * LD * 2, PT = CH * PLD * 2;
    static constexpr int SUMS = CH * D * 4 > 2 * TILE ? CH * D * 4 : 2 * TILE;           // log decays, then G and H
    static constexpr int LDM = 24;                                       // row stride of the inverses of the diagonal blocks
    static constexpr int SMEM = 5 * TILE + SUMS + 4 * PT + CH * 17 * 4 + CH * LDM * 2;
};

// acc (16 rows from m0) += A B with a lower triangular A (blocks of 16): B stored [k][n]
template <int NTL>
__device__ __forceinline__ void lower_gemm(float (&acc)[NTL][4], const bf16* A, int m0, const bf16* B, int ldb, int n0) {
    for (int k0 = 0; k0 <= m0; k0 += 16) {
        uint32_t p[4];
        load_a(p, A, PLD, m0, k0);
#pragma unroll
        for (int t = 0; t < NTL; t += 2) {
            uint32_t b[4];
            load_b2_t(b, B, ldb, n0 + t * 8, k0);
            mma16816(acc[t], p, b[0], b[1]);
            mma16816(acc[t + 1], p, b[2], b[3]);
        }
    }
}

// grid (chunks, H)
template <int D>
__global__ void __launch_bounds__(NT, D == 64 ? 2 : 1) delta_chunk_kernel(Args a, int chunks) {
    using C = Cfg<D>;
    constexpr int LD = C::LD, LDM = C::LDM, SEG = C::SEG, HT = D / 16;      // HT: n-tiles of a warp's half of D columns
    extern __shared__ __align__(16) unsigned char smem[];
    bf16* U = reinterpret_cast<bf16*>(smem);                 // [CH][LD] each
    bf16* B = U + CH * LD;
    bf16* K = B + CH * LD;
    bf16* R = K + CH * LD;
    bf16* V = R + CH * LD;
    unsigned char* sums = smem + 5 * C::TILE;
    float* Lw = reinterpret_cast<float*>(sums);              // [CH][D] log decays summed inside a segment
    bf16* G = reinterpret_cast<bf16*>(sums);                 // [CH][LD]
    bf16* H = G + CH * LD;                                   // [CH][LD]
    bf16* UB = reinterpret_cast<bf16*>(sums + C::SUMS);      // [CH][PLD] tril(U B^T, -1)
    bf16* UK = UB + CH * PLD;                                // [CH][PLD] tril(U K^T, -1)
    bf16* RB = UK + CH * PLD;                                // [CH][PLD] tril(R B^T)
    bf16* RK = RB + CH * PLD;                                // [CH][PLD] tril(R K^T)
    float* A = reinterpret_cast<float*>(RK + CH * PLD);      // [CH][17] the diagonal blocks of tril(U B^T, -1)
    bf16* M = reinterpret_cast<bf16*>(A + CH * 17);          // [CH][LDM] and the inverses of I plus them
    __shared__ float inv[CH], seg[C::SEGS][D], whole[D];
    const int* it = a.groups + blockIdx.x * G_INTS;
    const int h = blockIdx.y, row0 = it[G_ROW], n = it[G_N], d = a.d;
    const int w = threadIdx.x >> 5, l = threadIdx.x & 31, g = l >> 2, q = l & 3;
    // this warp's rows and columns of a D-wide product; the two warps of a scheduler share the work of triangular ones evenly
    const int half = w >> 2, m0 = 16 * (half ? 3 - (w & 3) : w & 3), n0 = half * (D / 2);
    const bf16* z = (const bf16*)a.z + (long long)row0 * a.ldz + h * d;
    load_rows<D, LD>(K, z + a.zk, a.ldz, n, d);
    load_rows<D, LD>(R, z + a.zr, a.ldz, n, d);
    load_rows<D, LD>(V, z + a.zv, a.ldz, n, d);
    load_rows<D, LD>(B, z + a.za, a.ldz, n, d);
    cp_async_commit();
    {
        const int c = threadIdx.x % D, s = threadIdx.x / D, t0 = s * SEG;
        const float* wl = a.w + (long long)row0 * a.ldw + h * d + c;
        const float w0 = c < d ? a.w0[h * d + c] : 0.f;
        float x[SEG], sum = 0.f;
#pragma unroll
        for (int t = 0; t < SEG; ++t) x[t] = c < d && t0 + t < n ? wl[(t0 + t) * a.ldw] : 0.f;
#pragma unroll
        for (int t = 0; t < SEG; ++t) {
            sum += c < d && t0 + t < n ? -DECAY * sigmoid(x[t] + w0) : 0.f;
            Lw[(t0 + t) * D + c] = sum;
        }
        seg[s][c] = sum;
    }
    cp_async_wait<0>();
    __syncthreads();
    for (int t = w; t < CH; t += NT / 32) {
        float s = 0.f;
        for (int c = 2 * l; c < D; c += 64) {
            const float2 k = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(K + t * LD + c));
            s += k.x * k.x + k.y * k.y;
        }
        s = warp_sum(s);
        if (l == 0) inv[t] = rsqrtf(s + UNIT_EPS);
    }
    if (threadIdx.x < D) {                                   // in front of a segment, and the whole chunk
        float s = 0.f;
        for (int i = 0; i < C::SEGS; ++i) {
            const float x = seg[i][threadIdx.x];
            seg[i][threadIdx.x] = s;
            s += x;
        }
        whole[threadIdx.x] = __expf(s);
    }
    __syncthreads();
    for (int i = threadIdx.x; i < CH * (D / 2); i += NT) {
        const int t = i / (D / 2), c = i % (D / 2) * 2, at = t * LD + c;
        const float2 pre = *reinterpret_cast<const float2*>(&seg[t / SEG][c]);
        float2 L = *reinterpret_cast<const float2*>(Lw + t * D + c), P = pre;           // up to this token, and in front of it
        L.x += pre.x, L.y += pre.y;
        if (t % SEG) {
            const float2 x = *reinterpret_cast<const float2*>(Lw + (t - 1) * D + c);
            P.x += x.x, P.y += x.y;
        }
        const float2 k = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(K + at)), r = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(R + at)),
                     e = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(B + at));
        const float2 bias = c < d ? *reinterpret_cast<const float2*>(a.a_bias + h * d + c) : make_float2(0.f, 0.f);
        const float f = inv[t], ux = k.x * f, uy = k.y * f, nx = __expf(-L.x), ny = __expf(-L.y);
        *reinterpret_cast<__nv_bfloat162*>(U + at) = __floats2bfloat162_rn(ux * __expf(P.x), uy * __expf(P.y));
        *reinterpret_cast<__nv_bfloat162*>(B + at) = __floats2bfloat162_rn(ux * sigmoid(e.x + bias.x) * nx, uy * sigmoid(e.y + bias.y) * ny);
        *reinterpret_cast<__nv_bfloat162*>(K + at) = __floats2bfloat162_rn(k.x * nx, k.y * ny);
        *reinterpret_cast<__nv_bfloat162*>(R + at) = __floats2bfloat162_rn(r.x * __expf(L.x), r.y * __expf(L.y));
    }
    __syncthreads();
    {                                                        // scores: rows of U (warps 0 .. 3) or R against the rows of B and K up to them
        const bf16* rows = half ? R : U;
#pragma unroll
        for (int other = 0; other < 2; ++other) {
            float s[8][4];
            zero_acc<8>(s);
#pragma unroll
            for (int k0 = 0; k0 < D; k0 += 16) {
                uint32_t p[4];
                load_a(p, rows, LD, m0, k0);
#pragma unroll
                for (int t = 0; t < 8; t += 2)
                    if (8 * t <= m0) {
                        uint32_t b[4];
                        load_b2(b, other ? K : B, LD, t * 8, k0);
                        mma16816(s[t], p, b[0], b[1]);
                        mma16816(s[t + 1], p, b[2], b[3]);
                    }
            }
            bf16* to = half ? other ? RK : RB : other ? UK : UB;
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int i = m0 + g + 8 * e;
#pragma unroll
                for (int t = 0; t < 8; ++t)
                    if (8 * t <= m0 + 8) {
                        const int j = 8 * t + 2 * q;
                        const float x = (half ? i >= j : i > j) ? s[t][2 * e] : 0.f, y = (half ? i >= j + 1 : i > j + 1) ? s[t][2 * e + 1] : 0.f;
                        *reinterpret_cast<__nv_bfloat162*>(to + i * PLD + j) = __floats2bfloat162_rn(x, y);
                        if (!half && !other && j >= m0) A[i * 17 + j - m0] = x, A[i * 17 + j + 1 - m0] = y;
                    }
            }
        }
    }
    __syncthreads();
    if (threadIdx.x < CH) {                                  // inverses of the diagonal blocks of 16, a thread per column
        const int b = threadIdx.x & ~15, c = threadIdx.x & 15;
        float m[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            float s0 = 0.f, s1 = 0.f;
#pragma unroll
            for (int k = 0; k < i; ++k) (k & 1 ? s1 : s0) += A[(b + i) * 17 + k] * m[k];
            m[i] = i == c ? 1.f : -(s0 + s1);                // (zero in front of the diagonal)
        }
#pragma unroll
        for (int i = 0; i < 16; ++i) M[(b + i) * LDM + c] = __float2bfloat16(m[i]);
    }
    __syncthreads();
    // G and H, 16 columns at a time from the first block of rows to the last: block i is M_ii times what is left of its right side when the
    // blocks before it are known.  Warps 0 .. 3 have the columns of G, the others those of H (D = 128: two turns).
    for (int strip = w & 3; strip < D / 16; strip += 4) {
        bf16* X = half ? H : G;
        const int c0 = strip * 16;
        for (int i0 = 0; i0 < CH; i0 += 16) {
            float x[2][4], y[2][4];
            zero_acc<2>(x);
            zero_acc<2>(y);
            if (half) {
                lower_gemm<2>(y, UK, i0, V, LD, c0);
            } else {
#pragma unroll
                for (int t = 0; t < 2; ++t)
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        const float2 u = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(U + (i0 + g + 8 * e) * LD + c0 + 8 * t + 2 * q));
                        y[t][2 * e] = u.x, y[t][2 * e + 1] = u.y;
                    }
            }
            for (int k0 = 0; k0 < i0; k0 += 16) {
                uint32_t p[4], b[4];
                load_a(p, UB, PLD, i0, k0);
                load_b2_t(b, X, LD, c0, k0);
                mma16816(x[0], p, b[0], b[1]);
                mma16816(x[1], p, b[2], b[3]);
            }
#pragma unroll
            for (int t = 0; t < 2; ++t)
#pragma unroll
                for (int e = 0; e < 4; ++e) y[t][e] -= x[t][e];
            store_acc_bf16<2>(y, X, LD, i0, c0);
            __syncwarp();
            uint32_t p[4], b[4];
            load_a(p, M, LDM, i0, 0);
            load_b2_t(b, X, LD, c0, i0);
            zero_acc<2>(x);
            mma16816(x[0], p, b[0], b[1]);
            mma16816(x[1], p, b[2], b[3]);
            __syncwarp();
            store_acc_bf16<2>(x, X, LD, i0, c0);
            __syncwarp();
        }
    }
    __syncthreads();
    const Work<D> out(a.work, (long long)chunks * a.H, (long long)blockIdx.x * a.H + h);
    {
        float x[HT][4];
        zero_acc<HT>(x);
        lower_gemm<HT>(x, RB, m0, G, LD, n0);
#pragma unroll
        for (int t = 0; t < HT; ++t)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int i = m0 + g + 8 * e, c = n0 + 8 * t + 2 * q;
                const float2 r = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(R + i * LD + c));
                *reinterpret_cast<__nv_bfloat162*>(out.Q + i * D + c) = __floats2bfloat162_rn(r.x - x[t][2 * e], r.y - x[t][2 * e + 1]);
            }
        float y[HT][4];
        zero_acc<HT>(x);
        zero_acc<HT>(y);
        lower_gemm<HT>(x, RB, m0, H, LD, n0);
        lower_gemm<HT>(y, RK, m0, V, LD, n0);
#pragma unroll
        for (int t = 0; t < HT; ++t)
#pragma unroll
            for (int e = 0; e < 2; ++e)
                *reinterpret_cast<float2*>(out.N + (m0 + g + 8 * e) * D + n0 + 8 * t + 2 * q) = make_float2(y[t][2 * e] - x[t][2 * e], y[t][2 * e + 1] - x[t][2 * e + 1]);
    }
    for (int rb = w & 3; rb < D / 16; rb += 4) {
        const int r0 = 16 * rb;
        float x[HT][4], y[HT][4];
        zero_acc<HT>(x);
        warp_gemm<HT, CH, true, true>(x, B, LD, r0, G, LD, n0);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int i = r0 + g + 8 * e;
            const float f = whole[i];
#pragma unroll
            for (int t = 0; t < HT; ++t)
                *reinterpret_cast<__nv_bfloat162*>(out.E + i * D + n0 + 8 * t + 2 * q) = __floats2bfloat162_rn(f * x[t][2 * e], f * x[t][2 * e + 1]);
        }
        zero_acc<HT>(x);
        zero_acc<HT>(y);
        warp_gemm<HT, CH, true, true>(x, B, LD, r0, H, LD, n0);
        warp_gemm<HT, CH, true, true>(y, K, LD, r0, V, LD, n0);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int i = r0 + g + 8 * e;
            const float f = whole[i];
#pragma unroll
            for (int t = 0; t < HT; ++t)
                *reinterpret_cast<float2*>(out.Dm + i * D + n0 + 8 * t + 2 * q) = make_float2(f * (y[t][2 * e] - x[t][2 * e]), f * (y[t][2 * e + 1] - x[t][2 * e + 1]));
        }
    }
    if (threadIdx.x < D) out.decay[threadIdx.x] = whole[threadIdx.x];
}

// ------------------------------------------------------------------------------------------------------- over the chunks
constexpr int PT = 128, COLS = 32, LDS = COLS + 8, STAGES = 3;

template <int D> struct Pass {
    static constexpr int LD = D + 8, LDF = COLS + 4;
    static constexpr int STAGE = D * LD * 2 + D * LDF * 4 + D * 4;       // E, a slice of D, e^L
    static constexpr int SMEM = STAGES * STAGE + D * LDS * 2;
};

// grid (D / 32, H, requests)
template <int D>
__global__ void __launch_bounds__(PT) delta_pass_kernel(Args a, int chunks) {
    using C = Pass<D>;
    constexpr int RB = D / 64;                               // blocks of 16 rows of the state per warp
    extern __shared__ __align__(16) unsigned char smem[];
    bf16* Sb = reinterpret_cast<bf16*>(smem + STAGES * C::STAGE);        // [D][LDS] the state in front of the chunk
    const int* it = a.groups + (chunks + blockIdx.z) * G_INTS;
    const int c0 = blockIdx.x * COLS, h = blockIdx.y, first = it[Q_FIRST], count = it[Q_CHUNKS], d = a.d;
    if (c0 >= d) return;
    const int w = threadIdx.x >> 5, l = threadIdx.x & 31, g = l >> 2, q = l & 3;
    const long long all = (long long)chunks * a.H;
    float* own = a.state == nullptr ? nullptr : a.state + ((long long)it[Q_SLOT] * a.H + h) * d * d;
    auto E = [&](int s) { return reinterpret_cast<bf16*>(smem + s * C::STAGE); };
    auto Dm = [&](int s) { return reinterpret_cast<float*>(smem + s * C::STAGE + D * C::LD * 2); };
    auto decay = [&](int s) { return Dm(s) + D * C::LDF; };
    auto load = [&](int i) {
        if (i < count) {
            const Work<D> in(a.work, all, (long long)(first + i) * a.H + h);
            const int s = i % STAGES;
            for (int k = threadIdx.x; k < D * (D / 8); k += PT) cp_async16(E(s) + k / (D / 8) * C::LD + k % (D / 8) * 8, in.E + k * 8, true);
            for (int k = threadIdx.x; k < D * (COLS / 4); k += PT)
                cp_async16(Dm(s) + k / (COLS / 4) * C::LDF + k % (COLS / 4) * 4, in.Dm + k / (COLS / 4) * D + c0 + k % (COLS / 4) * 4, true);
            if (threadIdx.x < D / 4) cp_async16(decay(s) + threadIdx.x * 4, in.decay + threadIdx.x * 4, true);
        }
        cp_async_commit();
    };
    for (int i = 0; i < STAGES - 1; ++i) load(i);
    float S[RB][4][4];
    const bool past = (it[Q_FLAGS] & 4) && own != nullptr;
#pragma unroll
    for (int b = 0; b < RB; ++b)
#pragma unroll
        for (int t = 0; t < 4; ++t)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int r = (w * RB + b) * 16 + g + 8 * e, c = c0 + 8 * t + 2 * q;
                const float2 x = past && r < d && c < d ? *reinterpret_cast<const float2*>(own + (long long)r * d + c) : make_float2(0.f, 0.f);
                S[b][t][2 * e] = x.x, S[b][t][2 * e + 1] = x.y;
            }
    for (int i = 0; i < count; ++i) {
        const int s = i % STAGES;
        cp_async_wait<STAGES - 2>();
        __syncthreads();                                     // this chunk's tiles are there, nobody reads Sb any more
        load(i + STAGES - 1);
#pragma unroll
        for (int b = 0; b < RB; ++b) store_acc_bf16<4>(S[b], Sb, LDS, (w * RB + b) * 16, 0);
        __syncthreads();
        const Work<D> out(a.work, all, (long long)(first + i) * a.H + h);
        for (int k = threadIdx.x; k < D * (COLS / 8); k += PT)
            *reinterpret_cast<uint4*>(out.S + k / (COLS / 8) * D + c0 + k % (COLS / 8) * 8) = *reinterpret_cast<const uint4*>(Sb + k / (COLS / 8) * LDS + k % (COLS / 8) * 8);
#pragma unroll
        for (int b = 0; b < RB; ++b) {
            const int m0 = (w * RB + b) * 16;
            float x[4][4];
            zero_acc<4>(x);
            warp_gemm<4, D, false, true>(x, E(s), C::LD, m0, Sb, LDS, 0);
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int r = m0 + g + 8 * e;
                const float f = decay(s)[r];
#pragma unroll
                for (int t = 0; t < 4; ++t) {
                    const float2 y = *reinterpret_cast<const float2*>(Dm(s) + r * C::LDF + 8 * t + 2 * q);
                    S[b][t][2 * e] = f * S[b][t][2 * e] - x[t][2 * e] + y.x;
                    S[b][t][2 * e + 1] = f * S[b][t][2 * e + 1] - x[t][2 * e + 1] + y.y;
                }
            }
        }
    }
    cp_async_wait<0>();
    if (own == nullptr) return;
#pragma unroll
    for (int b = 0; b < RB; ++b)
#pragma unroll
        for (int t = 0; t < 4; ++t)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int r = (w * RB + b) * 16 + g + 8 * e, c = c0 + 8 * t + 2 * q;
                if (r < d && c < d) *reinterpret_cast<float2*>(own + (long long)r * d + c) = make_float2(S[b][t][2 * e], S[b][t][2 * e + 1]);
            }
}

// ------------------------------------------------------------------------------------------------------------------- outputs
template <int D> constexpr int out_smem() { return (2 * CH + D) * (D + 8) * 2; }

// grid (chunks, H)
template <int D>
__global__ void __launch_bounds__(NT) delta_out_kernel(Args a, int chunks) {
    constexpr int LD = D + 8, HT = D / 16;
    extern __shared__ __align__(16) unsigned char smem[];
    bf16* Q = reinterpret_cast<bf16*>(smem);                 // [CH][LD]
    bf16* S = Q + CH * LD;                                   // [D][LD]
    bf16* G = S + D * LD;                                    // [CH][LD] gate, then the output
    __shared__ float red[2][CH];
    const int* it = a.groups + blockIdx.x * G_INTS;
    const int h = blockIdx.y, row0 = it[G_ROW], n = it[G_N], d = a.d;
    const int w = threadIdx.x >> 5, l = threadIdx.x & 31, g = l >> 2, q = l & 3;
    const int m0 = 16 * (w & 3), n0 = (w >> 2) * (D / 2);
    const Work<D> in(a.work, (long long)chunks * a.H, (long long)blockIdx.x * a.H + h);
    load_rows<D, LD>(Q, in.Q, D, CH, D);
    for (int i = threadIdx.x; i < D * (D / 8); i += NT) cp_async16(S + i / (D / 8) * LD + i % (D / 8) * 8, in.S + i * 8, i % (D / 8) * 8 < d);
    cp_async_commit();
    load_rows<D, LD>(G, (const bf16*)a.z + (long long)row0 * a.ldz + a.zg + h * d, a.ldz, n, d);
    cp_async_commit();
    float o[HT][4];
#pragma unroll
    for (int t = 0; t < HT; ++t)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const float2 x = *reinterpret_cast<const float2*>(in.N + (m0 + g + 8 * e) * D + n0 + 8 * t + 2 * q);
            o[t][2 * e] = x.x, o[t][2 * e + 1] = x.y;
        }
    cp_async_wait<1>();
    __syncthreads();
    warp_gemm<HT, D, false, true>(o, Q, LD, m0, S, LD, n0);
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        float y = 0.f;
#pragma unroll
        for (int t = 0; t < HT; ++t) y += o[t][2 * e] * o[t][2 * e] + o[t][2 * e + 1] * o[t][2 * e + 1];
        y += __shfl_xor_sync(0xffffffffu, y, 1);
        y += __shfl_xor_sync(0xffffffffu, y, 2);
        if (q == 0) red[w >> 2][m0 + g + 8 * e] = y;
    }
    cp_async_wait<0>();
    __syncthreads();
#pragma unroll
    for (int t = 0; t < HT; ++t) {
        const int c = n0 + 8 * t + 2 * q;
        const float2 k = c < d ? *reinterpret_cast<const float2*>(a.norm + h * d + c) : make_float2(0.f, 0.f);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int i = m0 + g + 8 * e;
            const float r = rsqrtf((red[0][i] + red[1][i]) / a.nd + a.eps);
            __nv_bfloat162* p = reinterpret_cast<__nv_bfloat162*>(G + i * LD + c);
            const float2 f = __bfloat1622float2(*p);
            *p = __floats2bfloat162_rn(o[t][2 * e] * r * k.x * sigmoid(f.x), o[t][2 * e + 1] * r * k.y * sigmoid(f.y));
        }
    }
    __syncthreads();
    bf16* out = (bf16*)a.out + (long long)row0 * a.ldo + h * d;
    for (int i = threadIdx.x; i < CH * (D / 8); i += NT) {
        const int r = i / (D / 8), c = i % (D / 8) * 8;
        if (r < n && c < d) *reinterpret_cast<uint4*>(out + (long long)r * a.ldo + c) = *reinterpret_cast<const uint4*>(G + r * LD + c);
    }
}

template <int D>
static int launch(const Args& a, int chunks, int requests, cudaStream_t st) {
    static_assert(Cfg<D>::SMEM <= 225 * 1024 && Pass<D>::SMEM <= 225 * 1024, "shared memory of one CTA");
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(delta_chunk_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg<D>::SMEM);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(delta_pass_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, Pass<D>::SMEM);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(delta_out_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, out_smem<D>());
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    delta_chunk_kernel<D><<<dim3(chunks, a.H), NT, Cfg<D>::SMEM, st>>>(a, chunks);
    delta_pass_kernel<D><<<dim3(D / COLS, a.H, requests), PT, Pass<D>::SMEM, st>>>(a, chunks);
    delta_out_kernel<D><<<dim3(chunks, a.H), NT, out_smem<D>(), st>>>(a, chunks);
    return (int)cudaGetLastError();
}

}  // namespace dltc
}  // namespace lmoe

using namespace lmoe;

// bytes of `work` for a chunk of a head of size d
LMOE_API long long lmoe_delta_tc_work(int d) {
    const long long D = d <= 64 ? 64 : 128;
    return 4 * (64 * D + D * D + D) + 2 * (64 * D + 2 * D * D);
}

// bf16; head size a multiple of 16 up to 128, pitches and first columns multiples of 8, 16-byte bases.  a.groups [chunks + requests, 8]: chunks of up
// to 64 tokens (only a request's last one is shorter), then the requests (slot, flags, first chunk, chunks).
LMOE_API int lmoe_delta_tc(const dlt::Args* ap, int chunks, int requests, cudaStream_t st) {
    const dlt::Args& a = *ap;
    if (chunks <= 0 || requests <= 0 || requests > 65535 || a.H <= 0 || a.H > 65535 || a.d <= 0 || a.d > 128 || a.d % 16 || a.nd <= 0 || a.ldz % 8 || a.ldo % 8 ||
        ((a.zr | a.zk | a.zv | a.za | a.zg) & 7) || a.groups == nullptr || a.work == nullptr || a.w == nullptr ||
        ((reinterpret_cast<uintptr_t>(a.z) | reinterpret_cast<uintptr_t>(a.out) | reinterpret_cast<uintptr_t>(a.state) | reinterpret_cast<uintptr_t>(a.work)) & 15))
        return -1;
    return a.d <= 64 ? dltc::launch<64>(a, chunks, requests, st) : dltc::launch<128>(a, chunks, requests, st);
}
