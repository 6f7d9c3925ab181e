// State-space duality over prompts for bf16 (mathematics and arguments: ssd.cu, ssd.cuh), state and head sizes up to 128: chunks of 64 tokens
// on tensor-core fragments (mma.sync), an fp32 state in registers.  With L_i the sum of the log decays of a chunk up to token i,
//     P_ij = (C_i . B_j) e^{L_i - L_j} dt_j [i >= j],   y = P X + e^{L_i} C S + D x,   S <- e^{L_n} S + (e^{L_n - L_j} dt_j B_j)^T X
// Requests are cut into groups of chunks so that (group, head) pairs fill the GPU:
//   ssd_state_kernel     what a group adds to the state and its log decay, for groups that are not their request's last one
//   ssd_combine_kernel   those sums -> the state in front of every group
//   ssd_out_kernel       outputs, each group from the state in front of it; a request's last group leaves the new state
// A request of one group needs the last kernel only.  Decays and step sizes are fp32; B and the scores are rounded once, behind them.
#include "chunk_state.cuh"
#include "ssd.cuh"

namespace lmoe {
namespace ssdt {
using namespace chk;
using namespace rt;
using ssd::Args;

template <int DK, int DV> struct Cfg : Shape<DK, DV> {
    using S = Shape<DK, DV>;
    static constexpr int STATE_SMEM = 2 * S::KV;
    static constexpr int OUT_SMEM = 2 * S::KV + CH * S::LDK * 2 + DK * S::LDV * 2 + CH * PLD * 2 + CH * S::LDV * 2;
};

// a chunk's step sizes and the running sums of its log decays, two tokens per lane of one warp; tokens that are not there: 0
__device__ __forceinline__ void chunk_steps(const Args& a, long long row, int n, int h, float* dt, float* L) {
    const int l = threadIdx.x & 31, i = 2 * l;
    const long long at = row * a.H + h;
    const float d0 = i < n ? a.dt[at + (long long)i * a.H] : 0.f, d1 = i + 1 < n ? a.dt[at + (long long)(i + 1) * a.H] : 0.f;
    const float g0 = i < n ? a.la[at + (long long)i * a.H] : 0.f, g1 = i + 1 < n ? a.la[at + (long long)(i + 1) * a.H] : 0.f;
    float s = g0 + g1;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const float x = __shfl_up_sync(0xffffffffu, s, o);
        if (l >= o) s += x;
    }
    dt[i] = d0, dt[i + 1] = d1;
    L[i] = s - g1, L[i + 1] = s;
}

// grid (groups, H); groups without a place behind them have nothing to do
template <int DK, int DV>
__global__ void __launch_bounds__(NT) ssd_state_kernel(Args a) {
    using C = Cfg<DK, DV>;
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ float dt[2][CH], L[2][CH];
    const int* it = a.groups + blockIdx.x * G_INTS;
    const int h = blockIdx.y, row0 = it[G_ROW], n = it[G_N], to = it[G_OUT];
    if (to < 0) return;
    const bf16* x = (const bf16*)a.xbc + (long long)row0 * a.ldx;
    const int at_b = a.H * a.dv + h / (a.H / a.G) * a.dn;
    auto B = [&](int s) { return reinterpret_cast<bf16*>(smem + s * C::KV); };
    auto X = [&](int s) { return B(s) + CH * C::LDK; };
    auto load = [&](int t0) {
        const int s = t0 / CH & 1;
        load_rows<DK, C::LDK>(B(s), x + t0 * a.ldx + at_b, a.ldx, n - t0, a.dn);
        load_rows<DV, C::LDV>(X(s), x + t0 * a.ldx + h * a.dv, a.ldx, n - t0, a.dv);
        if (threadIdx.x < 32) chunk_steps(a, row0 + t0, n - t0, h, dt[s], L[s]);
    };
    State<DK, DV> S;
    S.load(nullptr, a.dn, a.dv);
    float total = 0.f;
    load(0);
    cp_async_commit();
    for (int t0 = 0; t0 < n; t0 += CH) {
        const int s = t0 / CH & 1;
        if (t0 + CH < n) load(t0 + CH);
        cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const float last = L[s][CH - 1];
        total += last;
        S.advance(B(s), X(s), __expf(last), [&](int j) { return __expf(last - L[s][j]) * dt[s][j]; });
        __syncthreads();
    }
    S.store(a.scratch + ((long long)to * a.H + h) * a.dn * a.dv, a.dn, a.dv);
    if (threadIdx.x == 0) a.decay[(long long)to * a.H + h] = total;
}

// grid (pieces, H, requests of several groups).  Places of a request: the state in front of its first group, then what every group but the
// last one adds, which becomes the state behind that group.
__global__ void __launch_bounds__(NT) ssd_combine_kernel(Args a) {
    const int* it = a.requests + blockIdx.z * G_INTS;
    const int h = blockIdx.y, size = a.dn * a.dv, e = (blockIdx.x * NT + threadIdx.x) * 4;
    if (e >= size) return;
    const long long first = it[R_STATE], next = (long long)a.H * size;
    float* at = a.scratch + (first * a.H + h) * size + e;
    float4 c = make_float4(0.f, 0.f, 0.f, 0.f);
    if ((it[R_FLAGS] & 4) && a.state != nullptr) c = load4(a.state + ((long long)it[R_SLOT] * a.H + h) * size + e);
    store4(at, c);
    for (int g = 1; g < it[R_GROUPS]; ++g) {
        const float4 m = load4(at + g * next);
        const float p = __expf(a.decay[(first + g) * a.H + h]);
        c = make_float4(p * c.x + m.x, p * c.y + m.y, p * c.z + m.z, p * c.w + m.w);
        store4(at + g * next, c);
    }
}

// grid (groups, H)
template <int DK, int DV>
__global__ void __launch_bounds__(NT, Cfg<DK, DV>::OUT_SMEM <= 110 * 1024 ? 2 : 1) ssd_out_kernel(Args a) {
    using F = Cfg<DK, DV>;
    extern __shared__ __align__(16) unsigned char smem[];
    bf16* C = reinterpret_cast<bf16*>(smem + 2 * F::KV);     // [CH][LDK] (one stage: it is not needed for long)
    bf16* Sb = C + CH * F::LDK;                              // [DK][LDV] the state in bf16
    bf16* P = Sb + DK * F::LDV;                              // [CH][PLD]
    bf16* Y = P + CH * PLD;                                  // [CH][LDV]
    __shared__ float dt[2][CH], L[2][CH];
    const int* it = a.groups + blockIdx.x * G_INTS;
    const int h = blockIdx.y, row0 = it[G_ROW], n = it[G_N], from = it[G_IN], flags = it[G_FLAGS];
    const int w = threadIdx.x >> 5, l = threadIdx.x & 31, g = l >> 2, q = l & 3;
    const int m0 = 16 * (w & 3), o_n0 = (w >> 2) * (DV / 2), a_n0 = (w >> 2) * 32;       // this warp's rows; columns of outputs and scores
    const bf16* x = (const bf16*)a.xbc + (long long)row0 * a.ldx;
    bf16* y = (bf16*)a.y + (long long)row0 * a.ldy + h * a.dv;
    const int at_b = a.H * a.dv + h / (a.H / a.G) * a.dn;
    const long long size = (long long)a.dn * a.dv;
    float* own = a.state == nullptr ? nullptr : a.state + ((long long)it[G_SLOT] * a.H + h) * size;
    const float D = a.d[h];
    auto B = [&](int s) { return reinterpret_cast<bf16*>(smem + s * F::KV); };
    auto X = [&](int s) { return B(s) + CH * F::LDK; };
    auto load_c = [&](int t0) { load_rows<DK, F::LDK>(C, x + t0 * a.ldx + at_b + a.G * a.dn, a.ldx, n - t0, a.dn); };
    auto load = [&](int t0) {
        const int s = t0 / CH & 1;
        const bf16* p = x + t0 * a.ldx;
        load_rows<DK, F::LDK>(B(s), p + at_b, a.ldx, n - t0, a.dn);
        load_rows<DV, F::LDV>(X(s), p + h * a.dv, a.ldx, n - t0, a.dv);
        if (threadIdx.x < 32) chunk_steps(a, row0 + t0, n - t0, h, dt[s], L[s]);
    };
    load(0);
    load_c(0);
    cp_async_commit();
    State<DK, DV> S;
    S.load(from >= 0 ? a.scratch + ((long long)from * a.H + h) * size : (flags & 4) ? own : nullptr, a.dn, a.dv);
    store_acc_bf16<F::S_NT>(S.s, Sb, F::LDV, S.m0, S.n0);
    for (int t0 = 0; t0 < n; t0 += CH) {
        const int s = t0 / CH & 1, nt = min(CH, n - t0);
        cp_async_wait<0>();
        __syncthreads();                                     // this chunk's tiles and Sb are there, the previous output has left Y
        if (t0 + CH < n) load(t0 + CH);
        cp_async_commit();
        float o[F::O_NT][4], z[4][4];
        zero_acc<F::O_NT>(o);
        zero_acc<4>(z);
        warp_gemm<F::O_NT, DK, false, true>(o, C, F::LDK, m0, Sb, F::LDV, o_n0);
        if (a_n0 <= m0 + 15) warp_gemm<4, DK, false, false>(z, C, F::LDK, m0, B(s), F::LDK, a_n0);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int i = m0 + g + 8 * e;
            const float Li = L[s][i], f = __expf(Li);
#pragma unroll
            for (int t = 0; t < F::O_NT; ++t) o[t][2 * e] *= f, o[t][2 * e + 1] *= f;
#pragma unroll
            for (int t = 0; t < 4; ++t) {
                const int j = a_n0 + 8 * t + 2 * q;
                const float y0 = i >= j ? z[t][2 * e] * __expf(Li - L[s][j]) * dt[s][j] : 0.f;
                const float y1 = i >= j + 1 ? z[t][2 * e + 1] * __expf(Li - L[s][j + 1]) * dt[s][j + 1] : 0.f;
                *reinterpret_cast<__nv_bfloat162*>(P + i * PLD + j) = __floats2bfloat162_rn(y0, y1);
            }
        }
        const float last = L[s][CH - 1];
        S.advance(B(s), X(s), __expf(last), [&](int j) { return __expf(last - L[s][j]) * dt[s][j]; });
        __syncthreads();                                     // P is complete, nobody reads Sb and C any more
        if (t0 + CH < n) load_c(t0 + CH);
        cp_async_commit();
        for (int k0 = 0; k0 <= m0; k0 += 16) {               // tokens behind row m0 + 15 are hidden
            uint32_t p[4];
            load_a(p, P, PLD, m0, k0);
#pragma unroll
            for (int t = 0; t < F::O_NT; t += 2) {
                uint32_t b[4];
                load_b2_t(b, X(s), F::LDV, o_n0 + t * 8, k0);
                mma16816(o[t], p, b[0], b[1]);
                mma16816(o[t + 1], p, b[2], b[3]);
            }
        }
        store_acc_bf16<F::S_NT>(S.s, Sb, F::LDV, S.m0, S.n0);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int i = m0 + g + 8 * e;
#pragma unroll
            for (int t = 0; t < F::O_NT; ++t) {
                const int c = o_n0 + 8 * t + 2 * q;
                const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(X(s) + i * F::LDV + c));
                *reinterpret_cast<__nv_bfloat162*>(Y + i * F::LDV + c) = __floats2bfloat162_rn(o[t][2 * e] + D * v.x, o[t][2 * e + 1] + D * v.y);
            }
        }
        __syncthreads();
        for (int i = threadIdx.x; i < CH * (DV / 8); i += NT) {
            const int r = i / (DV / 8), c = i % (DV / 8) * 8;
            if (r < nt && c < a.dv) *reinterpret_cast<uint4*>(y + (t0 + r) * a.ldy + c) = *reinterpret_cast<const uint4*>(Y + r * F::LDV + c);
        }
    }
    if ((flags & 2) && own != nullptr) S.store(own, a.dn, a.dv);
}

template <int DK, int DV>
static int launch(const Args& a, cudaStream_t st) {
    using C = Cfg<DK, DV>;
    static_assert(C::OUT_SMEM <= 225 * 1024, "shared memory of one CTA");
    cudaError_t e = cudaSuccess;
    if (a.m > 0) {
        e = cudaFuncSetAttribute(ssd_state_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::STATE_SMEM);
        if (e != cudaSuccess) return (int)e;
        ssd_state_kernel<DK, DV><<<dim3(a.n, a.H), NT, C::STATE_SMEM, st>>>(a);
        ssd_combine_kernel<<<dim3((a.dn * a.dv / 4 + NT - 1) / NT, a.H, a.m), NT, 0, st>>>(a);
    }
    e = cudaFuncSetAttribute(ssd_out_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::OUT_SMEM);
    if (e != cudaSuccess) return (int)e;
    ssd_out_kernel<DK, DV><<<dim3(a.n, a.H), NT, C::OUT_SMEM, st>>>(a);
    return (int)cudaGetLastError();
}

}  // namespace ssdt
}  // namespace lmoe

using namespace lmoe;

// bf16, y bf16; state and head sizes multiples of 16 up to 128, pitches multiples of 8, 16-byte bases.  a.groups [n, 8], a.requests [m, 8]
// (requests of several groups; their groups but the last one are whole chunks), a.scratch and a.decay for them.
LMOE_API int lmoe_ssd_tc(const ssd::Args* ap, cudaStream_t st) {
    const ssd::Args& a = *ap;
    if (a.n <= 0 || a.m < 0 || a.H <= 0 || a.G <= 0 || a.H % a.G || a.dn <= 0 || a.dv <= 0 || a.dn > 128 || a.dv > 128 || a.dn % 16 || a.dv % 16 || a.ldx % 8 || a.ldy % 8 ||
        a.y_f32 || a.groups == nullptr || a.dt == nullptr || a.la == nullptr || (a.m > 0 && (a.scratch == nullptr || a.decay == nullptr || a.requests == nullptr)) ||
        ((reinterpret_cast<uintptr_t>(a.xbc) | reinterpret_cast<uintptr_t>(a.y) | reinterpret_cast<uintptr_t>(a.state) | reinterpret_cast<uintptr_t>(a.scratch)) & 15))
        return -1;
    if (a.dn <= 64) return a.dv <= 64 ? ssdt::launch<64, 64>(a, st) : ssdt::launch<64, 128>(a, st);
    return a.dv <= 64 ? ssdt::launch<128, 64>(a, st) : ssdt::launch<128, 128>(a, st);
}
