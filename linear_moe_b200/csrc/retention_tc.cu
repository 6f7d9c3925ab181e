// Retention over prompts for bf16 (mathematics and arguments: retention.cu, retention.cuh), head sizes up to 128: chunks of 64 tokens on
// tensor-core fragments (mma.sync), an fp32 state in registers, norm and gate in the epilogue.  With p_n = decay^n and a chunk of n tokens,
//     A = (Q K^T) p_{i - j} [i >= j],   O = scale (A V + p_{i + 1} Q S),   S <- p_n S + (p_{n - 1 - j} K)^T V
// Requests are cut into groups of chunks so that (group, head) pairs fill the GPU:
//   retention_state_kernel     what a group adds to the state, for groups that are not their request's last one
//   retention_combine_kernel   those sums -> the state in front of every group
//   retention_out_kernel       outputs, each group from the state in front of it; a request's last group leaves the new state
// A request of one group needs the last kernel only.  The powers are fp32; keys and scores are rounded once, behind their decay.
#include "chunk_state.cuh"
#include "retention.cuh"

namespace lmoe {
namespace rtc {
using namespace chk;
using namespace rt;

template <int DK, int DV> struct Cfg : Shape<DK, DV> {
    using S = Shape<DK, DV>;
    static constexpr int STATE_SMEM = 2 * S::KV;
    static constexpr int OUT_SMEM = 2 * (S::KV + CH * S::LDK * 2) + CH * S::LDV * 2 + DK * S::LDV * 2 + CH * PLD * 2;
};

// adds a chunk of n tokens; pw: decay^0 ..
template <int DK, int DV>
__device__ __forceinline__ void advance(State<DK, DV>& S, const bf16* K, const bf16* V, const float* pw, int n) {
    S.advance(K, V, pw[n], [&](int j) { return pw[max(n - 1 - j, 0)]; });
}

// grid (groups, H); groups without a place behind them have nothing to do
template <int DK, int DV>
__global__ void __launch_bounds__(NT) retention_state_kernel(Args a) {
    using C = Cfg<DK, DV>;
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ float pw[CH + 1];
    const int* it = a.groups + blockIdx.x * G_INTS;
    const int h = blockIdx.y, row0 = it[G_ROW], n = it[G_N], to = it[G_OUT];
    if (to < 0) return;
    for (int i = threadIdx.x; i <= CH; i += NT) pw[i] = a.powers[h * (CH + 1) + i];
    const bf16* k = (const bf16*)a.z + (long long)row0 * a.ldz + a.zk + h * a.dk;
    const bf16* v = (const bf16*)a.z + (long long)row0 * a.ldz + a.zv + h * a.dv;
    auto K = [&](int s) { return reinterpret_cast<bf16*>(smem + s * C::KV); };
    auto V = [&](int s) { return K(s) + CH * C::LDK; };
    auto load = [&](int t0) {
        const int s = t0 / CH & 1;
        load_rows<DK, C::LDK>(K(s), k + t0 * a.ldz, a.ldz, n - t0, a.dk);
        load_rows<DV, C::LDV>(V(s), v + t0 * a.ldz, a.ldz, n - t0, a.dv);
    };
    State<DK, DV> S;
    S.load(nullptr, a.dk, a.dv);
    load(0);
    cp_async_commit();
    for (int t0 = 0; t0 < n; t0 += CH) {
        if (t0 + CH < n) load(t0 + CH);
        cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        advance(S, K(t0 / CH & 1), V(t0 / CH & 1), pw, min(CH, n - t0));
        __syncthreads();
    }
    S.store(a.scratch + ((long long)to * a.H + h) * a.dk * a.dv, a.dk, a.dv);
}

// grid (pieces, H, requests of several groups).  Places of a request: the state in front of its first group, then what every group but the
// last one adds, which becomes the state behind that group.
__global__ void __launch_bounds__(NT) retention_combine_kernel(Args a) {
    const int* it = a.requests + blockIdx.z * G_INTS;
    const int h = blockIdx.y, size = a.dk * a.dv, e = (blockIdx.x * NT + threadIdx.x) * 4;
    if (e >= size) return;
    const float p = (float)pow(a.decay[h], (double)it[R_TOKENS]);
    float* at = a.scratch + ((long long)it[R_STATE] * a.H + h) * size + e;
    const long long next = (long long)a.H * size;
    float4 c = make_float4(0.f, 0.f, 0.f, 0.f);
    if ((it[R_FLAGS] & 4) && a.state != nullptr) c = load4(a.state + ((long long)it[R_SLOT] * a.H + h) * size + e);
    store4(at, c);
    for (int g = 1; g < it[R_GROUPS]; ++g) {
        const float4 m = load4(at + g * next);
        c = make_float4(p * c.x + m.x, p * c.y + m.y, p * c.z + m.z, p * c.w + m.w);
        store4(at + g * next, c);
    }
}

// grid (groups, H)
template <int DK, int DV>
__global__ void __launch_bounds__(NT) retention_out_kernel(Args a) {
    using C = Cfg<DK, DV>;
    extern __shared__ __align__(16) unsigned char smem[];
    constexpr int STAGE = C::KV + CH * C::LDK * 2;
    bf16* G = reinterpret_cast<bf16*>(smem + 2 * STAGE);     // [CH][LDV] gate, then the output
    bf16* Sb = G + CH * C::LDV;                              // [DK][LDV] the state in bf16
    bf16* P = Sb + DK * C::LDV;                              // [CH][PLD]
    __shared__ float pw[CH + 1], red[2][CH];
    const int* it = a.groups + blockIdx.x * G_INTS;
    const int h = blockIdx.y, row0 = it[G_ROW], n = it[G_N], from = it[G_IN], flags = it[G_FLAGS];
    const int w = threadIdx.x >> 5, l = threadIdx.x & 31, g = l >> 2, q = l & 3;
    const int m0 = 16 * (w & 3), o_n0 = (w >> 2) * (DV / 2), a_n0 = (w >> 2) * 32;       // this warp's rows; columns of outputs and scores
    for (int i = threadIdx.x; i <= CH; i += NT) pw[i] = a.powers[h * (CH + 1) + i];
    const bf16* z = (const bf16*)a.z + (long long)row0 * a.ldz;
    bf16* out = (bf16*)a.out + (long long)row0 * a.ldo + h * a.dv;
    const long long size = (long long)a.dk * a.dv;
    float* own = a.state == nullptr ? nullptr : a.state + ((long long)it[G_SLOT] * a.H + h) * size;
    auto K = [&](int s) { return reinterpret_cast<bf16*>(smem + s * STAGE); };
    auto V = [&](int s) { return K(s) + CH * C::LDK; };
    auto Q = [&](int s) { return V(s) + CH * C::LDV; };
    auto load = [&](int t0) {
        const int s = t0 / CH & 1;
        const bf16* p = z + t0 * a.ldz;
        load_rows<DK, C::LDK>(Q(s), p + a.zq + h * a.dk, a.ldz, n - t0, a.dk);
        load_rows<DK, C::LDK>(K(s), p + a.zk + h * a.dk, a.ldz, n - t0, a.dk);
        load_rows<DV, C::LDV>(V(s), p + a.zv + h * a.dv, a.ldz, n - t0, a.dv);
    };
    load(0);
    cp_async_commit();
    State<DK, DV> S;
    S.load(from >= 0 ? a.scratch + ((long long)from * a.H + h) * size : (flags & 4) ? own : nullptr, a.dk, a.dv);
    store_acc_bf16<C::S_NT>(S.s, Sb, C::LDV, S.m0, S.n0);
    for (int t0 = 0; t0 < n; t0 += CH) {
        const int s = t0 / CH & 1, nt = min(CH, n - t0);
        cp_async_wait<0>();
        __syncthreads();                                     // this chunk's tiles and Sb are there, the previous output has left G
        load_rows<DV, C::LDV>(G, z + t0 * a.ldz + a.zg + h * a.dv, a.ldz, nt, a.dv);
        cp_async_commit();
        if (t0 + CH < n) load(t0 + CH);
        cp_async_commit();
        float o[C::O_NT][4], x[4][4];
        zero_acc<C::O_NT>(o);
        zero_acc<4>(x);
        warp_gemm<C::O_NT, DK, false, true>(o, Q(s), C::LDK, m0, Sb, C::LDV, o_n0);
        if (a_n0 <= m0 + 15) warp_gemm<4, DK, false, false>(x, Q(s), C::LDK, m0, K(s), C::LDK, a_n0);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int i = m0 + g + 8 * e;
            const float f = pw[i + 1] * a.scale;
#pragma unroll
            for (int t = 0; t < C::O_NT; ++t) o[t][2 * e] *= f, o[t][2 * e + 1] *= f;
#pragma unroll
            for (int t = 0; t < 4; ++t) {
                const int j = a_n0 + 8 * t + 2 * q;
                const float y0 = i >= j ? x[t][2 * e] * pw[max(i - j, 0)] * a.scale : 0.f;
                const float y1 = i >= j + 1 ? x[t][2 * e + 1] * pw[max(i - j - 1, 0)] * a.scale : 0.f;
                *reinterpret_cast<__nv_bfloat162*>(P + i * PLD + j) = __floats2bfloat162_rn(y0, y1);
            }
        }
        advance(S, K(s), V(s), pw, nt);
        __syncthreads();                                     // P is complete, nobody reads Sb any more
        for (int k0 = 0; k0 <= m0; k0 += 16) {               // keys behind row m0 + 15 are hidden
            uint32_t p[4];
            load_a(p, P, PLD, m0, k0);
#pragma unroll
            for (int t = 0; t < C::O_NT; t += 2) {
                uint32_t b[4];
                load_b2_t(b, V(s), C::LDV, o_n0 + t * 8, k0);
                mma16816(o[t], p, b[0], b[1]);
                mma16816(o[t + 1], p, b[2], b[3]);
            }
        }
        store_acc_bf16<C::S_NT>(S.s, Sb, C::LDV, S.m0, S.n0);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            float y = 0.f;
#pragma unroll
            for (int t = 0; t < C::O_NT; ++t) y += o[t][2 * e] * o[t][2 * e] + o[t][2 * e + 1] * o[t][2 * e + 1];
            y += __shfl_xor_sync(0xffffffffu, y, 1);
            y += __shfl_xor_sync(0xffffffffu, y, 2);
            if (q == 0) red[w >> 2][m0 + g + 8 * e] = y;
        }
        cp_async_wait<1>();                                  // the gate
        __syncthreads();
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int i = m0 + g + 8 * e;
            const float r = 1.f / sqrtf((red[0][i] + red[1][i]) / a.nv + a.eps);
#pragma unroll
            for (int t = 0; t < C::O_NT; ++t) {
                __nv_bfloat162* p = reinterpret_cast<__nv_bfloat162*>(G + i * C::LDV + o_n0 + 8 * t + 2 * q);
                const float2 f = __bfloat1622float2(*p);
                *p = __floats2bfloat162_rn(o[t][2 * e] * r * silu_f(f.x), o[t][2 * e + 1] * r * silu_f(f.y));
            }
        }
        __syncthreads();
        for (int i = threadIdx.x; i < CH * (DV / 8); i += NT) {
            const int r = i / (DV / 8), c = i % (DV / 8) * 8;
            if (r < nt && c < a.dv) *reinterpret_cast<uint4*>(out + (t0 + r) * a.ldo + c) = *reinterpret_cast<const uint4*>(G + r * C::LDV + c);
        }
    }
    if ((flags & 2) && own != nullptr) S.store(own, a.dk, a.dv);
}

template <int DK, int DV>
static int launch(const Args& a, cudaStream_t st) {
    using C = Cfg<DK, DV>;
    static_assert(C::OUT_SMEM <= 225 * 1024, "shared memory of one CTA");
    cudaError_t e = cudaSuccess;
    if (a.m > 0) {
        e = cudaFuncSetAttribute(retention_state_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::STATE_SMEM);
        if (e != cudaSuccess) return (int)e;
        retention_state_kernel<DK, DV><<<dim3(a.n, a.H), NT, C::STATE_SMEM, st>>>(a);
        retention_combine_kernel<<<dim3((a.dk * a.dv / 4 + NT - 1) / NT, a.H, a.m), NT, 0, st>>>(a);
    }
    e = cudaFuncSetAttribute(retention_out_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::OUT_SMEM);
    if (e != cudaSuccess) return (int)e;
    retention_out_kernel<DK, DV><<<dim3(a.n, a.H), NT, C::OUT_SMEM, st>>>(a);
    return (int)cudaGetLastError();
}

}  // namespace rtc
}  // namespace lmoe

using namespace lmoe;

// bf16; queries and keys rotated already; head sizes multiples of 16 up to 128, pitches and first columns multiples of 8, 16-byte bases.
// a.groups [n, 8], a.requests [m, 8] (requests of several groups; their groups but the last one are whole chunks), a.scratch for them.
LMOE_API int lmoe_retention_tc(const rt::Args* ap, cudaStream_t st) {
    const rt::Args& a = *ap;
    if (a.n <= 0 || a.m < 0 || a.H <= 0 || a.dk <= 0 || a.dv <= 0 || a.dk > 128 || a.dv > 128 || a.dk % 16 || a.dv % 16 || a.nv <= 0 || a.ldz % 8 || a.ldo % 8 ||
        ((a.zq | a.zk | a.zv | a.zg) & 7) || a.groups == nullptr || a.powers == nullptr || (a.m > 0 && (a.scratch == nullptr || a.requests == nullptr)) ||
        ((reinterpret_cast<uintptr_t>(a.z) | reinterpret_cast<uintptr_t>(a.out) | reinterpret_cast<uintptr_t>(a.state) | reinterpret_cast<uintptr_t>(a.scratch)) & 15))
        return -1;
    if (a.dk <= 64) return a.dv <= 64 ? rtc::launch<64, 64>(a, st) : rtc::launch<64, 128>(a, st);
    return a.dv <= 64 ? rtc::launch<128, 64>(a, st) : rtc::launch<128, 128>(a, st);
}
