// Causal attention over packed prompts on the 5th-generation tensor cores (bf16, head sizes up to 128 in multiples of 8),
// with an optional sliding window and an optional output gate:
//     o = sigmoid(gate) * softmax(q . k * scale) v          key j visible to query i when 0 <= i - j (< window)
// Queries, keys and values are rows of separate matrices (packed_attn.cuh); a work item is up to 128 queries of one request.
//
// One CTA = one work item of one head, warp roles as in flash_attn_tc.cu and chunk_attn_tc.cu:
//   warp 0      TMA producer: Q once, then K_j / V_j tiles of 128 keys through two 2-stage rings; only tiles inside the window
//   warp 1      MMA issuer: S_{j+1} = Q K_{j+1}^T before O += P_j V_j
//   warps 4..19 four warps per 32 query rows split the columns: one tensor-memory read of the scores, row maximum over the parts
//               (shared memory and a named barrier), P = exp2(S - m), bf16 pack into the 128-byte-swizzled P tile
// O accumulates in tensor memory over all key tiles.  The maximum a row is scaled by may lag behind the true one by LAG (in
// units of log2), so that P stays below 2^LAG; only when a row runs ahead of that is O multiplied in tensor memory.
// With `cross`, a query head's weights are applied to the values of every kv head (talking heads, which mix these results afterwards): a
// CTA takes as many kv heads as fit 256 columns of tensor memory, and the values come in stages of 64 keys.  Where the scores are known to
// be `bounded` (normed queries and keys), P = exp2(S) as it is: no maximum, no exchange between threads, and P goes back to tensor memory
// into the columns its scores came from, from where the value product reads it; the shared memory of the P tile holds more stages of
// values.
// Sigmoid weights (every visible pair by itself, o = mul * sum of sigmoid(q . k * scale + bias[h]) v) are bounded too and take that form, with
// value heads up to 256.
// Every mbarrier wait is bounded; on expiry the error word is set and the CTA drains and frees its tensor memory.
#include "attn_math.cuh"
#include "flash_tc_utils.cuh"
#include "packed_attn.cuh"

namespace lmoe {
namespace patc {
using namespace lmoe::fatc;
using pa::Prompt;

constexpr float LAG = 8.f;
enum Weights { LAGGING, BOUNDED_SOFTMAX, SIGMOID };

// DQ: key dims, DT: value columns of a CTA
template <int DQ, int DT, bool BOUNDED>
struct __align__(1024) Smem {
    static constexpr int VK = DT > 128 ? 64 : BN;           // keys per stage of values
    static constexpr int ST = DT > 128 && BOUNDED ? 4 : 2;               // stages of values
    uint8_t q[BM * DQ * 2];
    uint8_t k[2][BN * DQ * 2];
    uint8_t v[ST][VK * DT * 2];
    uint8_t p[BOUNDED ? 16 : BM * BN * 2];
    float mx[BOUNDED ? 1 : 2][BOUNDED ? 1 : SPLIT][BOUNDED ? 1 : BM];
    uint64_t q_full, k_full[2], k_empty[2], v_full[ST], v_empty[ST], s_full[2], pv_done, p_ready[2];
    uint32_t tmem_base;
    int abort_flag;
};

__device__ __forceinline__ void tmem_st16(uint32_t taddr, const uint32_t (&r)[16]) {
    asm volatile("tcgen05.st.sync.aligned.32x32b.x16.b32 [%16], {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15};"
                 :: "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),
                    "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(taddr) : "memory");
}
// D += A B with A in tensor memory: row r in lane r, two consecutive k per column
__device__ __forceinline__ void umma_ta(uint32_t tmem_d, uint32_t tmem_a, uint32_t b_lo, uint32_t idesc, uint32_t accumulate, uint32_t issue) {
    asm volatile("{\n.reg .pred p, q;\n.reg .b64 db;\nsetp.ne.b32 p, %4, 0;\nsetp.ne.b32 q, %5, 0;\n"
                 "mov.b64 db, {%2, %6};\n"
                 "@q tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], db, %3, p;\n}"
                 :: "r"(tmem_d), "r"(tmem_a), "r"(b_lo), "r"(idesc), "r"(accumulate), "r"(issue), "r"(DESC_HI) : "memory");
}
__device__ __forceinline__ void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }

// DV: value dims of a head, NB: value heads of a CTA
template <int DQ, int DV, int NB, Weights W>
__global__ void __launch_bounds__(THREADS, 1)
packed_attn_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                      const __grid_constant__ CUtensorMap tmV, Prompt a) {
    extern __shared__ uint8_t smem_raw[];
    constexpr int DT = NB * DV;
    constexpr bool BOUNDED = W != LAGGING;
    using Sm = Smem<DQ, DT, BOUNDED>;
    constexpr int VK = Sm::VK, VS = BN / VK, ST = Sm::ST;   // VS: stages of values per tile of keys
    Sm& sm = *reinterpret_cast<Sm*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    constexpr int KQ = DQ / 64, KV = DT / 64;               // 64-element blocks along the head dimensions
    constexpr uint32_t TMEM_COLS = 512, O_COL = 2 * BN;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int* it = a.items + (long long)blockIdx.x * pa::I_N;
    const int row0 = it[pa::I_ROW], nq = it[pa::I_NQ], c0 = it[pa::I_C0], krow = it[pa::I_KROW];
    const int h = blockIdx.y, hk = h / (a.H / a.G), hv = a.cross ? blockIdx.z * NB : hk;       // hv: first value head
    const int nb_lo = a.window > 0 ? max(0, c0 - a.window + 1) / BN : 0;
    const int n_it = (c0 + nq + BN - 1) / BN - nb_lo;       // at least 1: a query sees its own key
    // bounded: a warp may be done with tile j + 1 while another one works on tile j, so neighbouring tiles have barriers of their own
    auto p_bar = [&](int j) { return &sm.p_ready[BOUNDED ? j & 1 : 0]; };
    auto p_phase = [](int j) { return (uint32_t)(BOUNDED ? (j >> 1) & 1 : j & 1); };
    volatile int* abort_flag = &sm.abort_flag;
    int* err = a.err;

    if (threadIdx.x == 0) {
        mbar_init(&sm.q_full, 1);
        for (int s = 0; s < 2; ++s) {
            mbar_init(&sm.k_full[s], 1); mbar_init(&sm.k_empty[s], 1);
            mbar_init(&sm.s_full[s], 1);
        }
        for (int s = 0; s < ST; ++s) { mbar_init(&sm.v_full[s], 1); mbar_init(&sm.v_empty[s], 1); }
        mbar_init(&sm.pv_done, 1);
        for (int s = 0; s < 2; ++s) mbar_init(&sm.p_ready[s], 4 * SPLIT);
        sm.abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" :: "r"(s32(&sm.tmem_base)), "r"(TMEM_COLS) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = sm.tmem_base;

    if (warp == 0) {
        if (lane == 0) {
            mbar_expect_tx(&sm.q_full, BM * DQ * 2);
#pragma unroll
            for (int kb = 0; kb < KQ; ++kb) tma_load_4d(sm.q + kb * BM * 128, &tmQ, &sm.q_full, kb * 64, h, row0, 0);
            for (int j = 0; j < n_it; ++j) {
                const int s = j & 1;
                const uint32_t ph = (j >> 1) & 1;
                const int key0 = krow + (nb_lo + j) * BN;
                if (!mbar_wait_suspend(&sm.k_empty[s], ph ^ 1, abort_flag, err, 0x7100 | s)) break;
                mbar_expect_tx(&sm.k_full[s], BN * DQ * 2);
#pragma unroll
                for (int kb = 0; kb < KQ; ++kb) tma_load_4d(sm.k[s] + kb * BN * 128, &tmK, &sm.k_full[s], kb * 64, hk, key0, 0);
                bool ok = true;
#pragma unroll
                for (int u = 0; u < VS; ++u) {
                    const int vi = j * VS + u, t = vi % ST;
                    ok = mbar_wait_suspend(&sm.v_empty[t], (vi / ST & 1) ^ 1, abort_flag, err, 0x7200 | t);
                    if (!ok) break;
                    mbar_expect_tx(&sm.v_full[t], VK * DT * 2);
#pragma unroll
                    for (int kk = 0; kk < VK / 64; ++kk)    // MN-major operand: per 64 keys, DT/64 boxes of {64 d, 64 keys}
#pragma unroll
                        for (int nb = 0; nb < KV; ++nb)     // (heads behind the last one read zeros)
                            tma_load_4d(sm.v[t] + (kk * KV + nb) * 8192, &tmV, &sm.v_full[t], nb % (DV / 64) * 64, hv + nb / (DV / 64),
                                        key0 + u * VK + kk * 64, 0);
                }
                if (!ok) break;
            }
        }
    } else if (warp == 1) {
        const uint32_t issue = lane == 0 ? 1u : 0u;
        constexpr uint32_t idesc_s = idesc_bf16<false, BN>();
        constexpr uint32_t idesc_o = idesc_bf16<true, DT>();
        bool ok = mbar_wait_suspend(&sm.q_full, 0, abort_flag, err, 0x8000);
        auto issue_s = [&](int j) -> bool {
            const int s = j & 1;
            if (!mbar_wait_suspend(&sm.k_full[s], (j >> 1) & 1, abort_flag, err, 0x8100 | s)) return false;
            tc_fence_after();
            const uint32_t ql = desc_lo<false>(s32(sm.q)), kl = desc_lo<false>(s32(sm.k[s]));
#pragma unroll
            for (int kk = 0; kk < DQ / UMMA_K; ++kk) {
                const uint32_t off = ((kk / 4) * (BM * 128) + (kk % 4) * 32) >> 4;
                umma_lo(tmem_base + s * BN, ql + off, kl + off, idesc_s, kk > 0 ? 1u : 0u, issue);
            }
            umma_commit_if(&sm.k_empty[s], issue);
            umma_commit_if(&sm.s_full[s], issue);
            return true;
        };
        if (ok) ok = issue_s(0);
        for (int j = 0; ok && j < n_it; ++j) {
            // score buffer (j + 1) & 1 was last read for P_{j-1}, whose p_ready was waited for in the previous iteration; with P_{j-1} in its
            // place, the product that reads it has to complete
            if (BOUNDED && j > 0 && j + 1 < n_it && !mbar_wait_suspend(&sm.pv_done, (j - 1) & 1, abort_flag, err, 0x8400)) break;
            if (j + 1 < n_it) { ok = issue_s(j + 1); if (!ok) break; }
#pragma unroll
            for (int u = 0; u < VS; ++u) {
                const int vi = j * VS + u, t = vi % ST;
                ok = mbar_wait_suspend(&sm.v_full[t], vi / ST & 1, abort_flag, err, 0x8200 | t);
                if (ok && u == 0) ok = mbar_wait_suspend(p_bar(j), p_phase(j), abort_flag, err, 0x8300);
                if (!ok) break;
                tc_fence_after();
                const uint32_t pl = BOUNDED ? tmem_base + (j & 1) * BN : desc_lo<false>(s32(sm.p)), vl = desc_lo<true>(s32(sm.v[t]));
#pragma unroll
                for (int kk = 0; kk < VK / UMMA_K; ++kk) {
                    const int kp = u * (VK / UMMA_K) + kk;  // 16-key step of the tile
                    const uint32_t aoff = ((kp / 4) * (BM * 128) + (kp % 4) * 32) >> 4;
                    const uint32_t boff = ((kk / 4) * (KV * 8192) + (kk % 4) * 2048) >> 4;
                    if (BOUNDED)                            // every 32 scores left 16 columns of P at their beginning
                        umma_ta(tmem_base + O_COL, pl + kp / 2 * 32 + kp % 2 * 8, vl + boff, idesc_o, (j > 0 || kp > 0) ? 1u : 0u, issue);
                    else umma_lo(tmem_base + O_COL, pl + aoff, vl + boff, idesc_o, (j > 0 || kp > 0) ? 1u : 0u, issue);
                }
                umma_commit_if(&sm.v_empty[t], issue);
            }
            if (!ok) break;
            umma_commit_if(&sm.pv_done, issue);
        }
    } else if (warp >= 4) {
        const int qd = warp & 3, part = (warp - 4) >> 2;
        const int r = qd * 32 + lane;                         // query row inside the tile
        const uint32_t lane_addr = tmem_base + ((uint32_t)(qd * 32) << 16);
        constexpr int CW = BN / SPLIT, OW = DT / SPLIT;       // score / output columns of this thread
        static_assert(CW == 32 && OW % 16 == 0, "tensor-memory load widths");
        const float sc = a.scale * LOG2E, lag = LAG / sc, head_bias = W == SIGMOID ? a.bias[h] * LOG2E : 0.f;
        uint8_t* prow = sm.p + ((part * CW) >> 6) * (BM * 128) + (r >> 3) * 1024 + (r & 7) * 128;
        const int ch0 = ((part * CW) & 63) >> 3;
        float m = -INFINITY, l = 0.f;
        bool alive = true;
        for (int j = 0; j < n_it; ++j) {
            const int s = j & 1, tile0 = (nb_lo + j) * BN;
            if (!mbar_wait_suspend(&sm.s_full[s], (j >> 1) & 1, abort_flag, err, 0x9100 | s)) { alive = false; break; }
            tc_fence_after();
            uint32_t v[CW];
            tmem_ld32(lane_addr + s * BN + part * CW, v);
            tmem_ld_wait();
            if (tile0 + BN - 1 > c0 || (a.window > 0 && tile0 <= c0 + BM - 1 - a.window)) {
                const int hi = c0 + r - (tile0 + part * CW);  // columns up to hi are not in the future
                const int lo = a.window > 0 ? hi - a.window : -1;
#pragma unroll
                for (int c = 0; c < CW; ++c)
                    if (c > hi || c <= lo) v[c] = W == SIGMOID && sc < 0.f ? 0x7f800000u : 0xff800000u;         // a weight of zero
            }
            if constexpr (!BOUNDED) {
                float mx4[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    mx4[e] = fmaxf(__uint_as_float(v[e]), __uint_as_float(v[e + 4]));
#pragma unroll
                    for (int c = 8; c < CW; c += 8) mx4[e] = max3(mx4[e], __uint_as_float(v[c + e]), __uint_as_float(v[c + e + 4]));
                }
                sm.mx[s][part][r] = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
                asm volatile("bar.sync %0, %1;" :: "r"(1 + qd), "n"(32 * SPLIT) : "memory");
                float mx = sm.mx[s][0][r];
#pragma unroll
                for (int p = 1; p < SPLIT; ++p) mx = fmaxf(mx, sm.mx[s][p][r]);
                // the four parts of a row see the same numbers and decide alike
                const bool grow = mx > m + lag;                   // also the first visible key of the row (m = -inf)
                const bool scaled = grow && m != -INFINITY;
                const float corr = scaled ? ex2((m - mx) * sc) : 1.f;
                if (grow) m = mx;
                l *= corr;
                if (__any_sync(0xffffffffu, scaled)) {            // not before tile 1: O holds something
                    if (!mbar_wait_suspend(&sm.pv_done, (j - 1) & 1, abort_flag, err, 0x9200)) { alive = false; break; }
                    tc_fence_after();
#pragma unroll
                    for (int c = 0; c < OW; c += 16) {
                        uint32_t o[16];
                        tmem_ld16(lane_addr + O_COL + part * OW + c, o);
                        tmem_ld_wait();
#pragma unroll
                        for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * corr);
                        tmem_st16(lane_addr + O_COL + part * OW + c, o);
                    }
                    tmem_st_wait();
                }
            }
            const float nm = W == SIGMOID ? -head_bias : BOUNDED || m == -INFINITY ? 0.f : -m * sc;
            const float2 sc2 = W == SIGMOID ? make_float2(-sc, -sc) : make_float2(sc, sc), nm2 = make_float2(nm, nm);
            float2 sum0 = make_float2(0.f, 0.f), sum1 = make_float2(0.f, 0.f);
#pragma unroll
            for (int c = 0; c < CW; c += 4) {
                const float2 x01 = __ffma2_rn(make_float2(__uint_as_float(v[c]), __uint_as_float(v[c + 1])), sc2, nm2);
                const float2 x23 = __ffma2_rn(make_float2(__uint_as_float(v[c + 2]), __uint_as_float(v[c + 3])), sc2, nm2);
                float p0 = ex2(x01.x), p1 = ex2(x01.y), p2 = ex2(x23.x), p3 = ex2(x23.y);
                if constexpr (W == SIGMOID) {                 // (hidden: 1 / infinity)
                    p0 = rcp(1.f + p0), p1 = rcp(1.f + p1), p2 = rcp(1.f + p2), p3 = rcp(1.f + p3);
                } else {
                    sum0 = __fadd2_rn(sum0, make_float2(p0, p1));
                    sum1 = __fadd2_rn(sum1, make_float2(p2, p3));
                }
                v[c >> 1] = pack_bf16(p0, p1);
                v[(c >> 1) + 1] = pack_bf16(p2, p3);
            }
            l += (sum0.x + sum0.y) + (sum1.x + sum1.y);
            if constexpr (BOUNDED) {
                uint32_t p[16];
#pragma unroll
                for (int c = 0; c < 16; ++c) p[c] = v[c];
                tmem_st16(lane_addr + s * BN + part * CW, p);
                tmem_st_wait();
                tc_fence_before();
            } else {
                // the P tile is free once O += P_{j-1} V_{j-1} has completed
                if (j > 0 && !mbar_wait_suspend(&sm.pv_done, (j - 1) & 1, abort_flag, err, 0x9300)) { alive = false; break; }
#pragma unroll
                for (int c = 0; c < 4; ++c)
                    *reinterpret_cast<uint4*>(prow + (((ch0 + c) ^ (r & 7)) << 4)) = make_uint4(v[4 * c], v[4 * c + 1], v[4 * c + 2], v[4 * c + 3]);
                tc_fence_before();
                asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            }
            __syncwarp();
            if (lane == 0) mbar_arrive(p_bar(j));
        }
        // (the product before the last one first: a barrier that is two phases behind looks like one that is done)
        if (BOUNDED && alive && n_it > 1) alive = mbar_wait_suspend(&sm.pv_done, (n_it - 2) & 1, abort_flag, err, 0x9500);
        if (alive) alive = mbar_wait_suspend(&sm.pv_done, (n_it - 1) & 1, abort_flag, err, 0x9400);
        tc_fence_after();
        float* ls = reinterpret_cast<float*>(sm.q);           // [SPLIT][BM]; every product has completed, the queries are not read any more
        ls[part * BM + r] = l;
        asm volatile("bar.sync %0, %1;" :: "r"(1 + qd), "n"(32 * SPLIT) : "memory");
        l = 0.f;
#pragma unroll
        for (int p = 0; p < SPLIT; ++p) l += ls[p * BM + r];
        uint32_t o[OW];
        if constexpr (OW == 48) {
#pragma unroll
            for (int c = 0; c < OW; c += 16) {
                uint32_t piece[16];
                tmem_ld16(lane_addr + O_COL + part * OW + c, piece);
                tmem_ld_wait();
#pragma unroll
                for (int i = 0; i < 16; ++i) o[c + i] = piece[i];
            }
        } else {
            tmem_ld<OW>(lane_addr + O_COL + part * OW, o);
            tmem_ld_wait();
        }
        if (alive && r < nq) {
            const float w = W == SIGMOID ? a.mul : 1.f / l;
            const long long row = row0 + r;
            const bf16* gp = a.gate == nullptr ? nullptr : (const bf16*)a.gate + row * a.ldg + h * a.dv;
#pragma unroll
            for (int c = 0; c < OW; c += 8) {
                const int col = (part * OW + c) % DV, nb = (part * OW + c) / DV;
                bf16* op = (bf16*)a.out + row * a.ldo + (long long)(a.cross ? h * a.G + hv + nb : h) * a.dv;
                if (col < a.dv && hv + nb < a.G) {
                    Vec<bf16> g, y;
                    if (gp != nullptr) g.load(gp + col);
#pragma unroll
                    for (int i = 0; i < 8; ++i) {
                        const float x = __uint_as_float(o[c + i]) * w;
                        y.set(i, gp != nullptr ? x * rcp(1.f + ex2(-LOG2E * g.get(i))) : x);
                    }
                    y.store(op + col);
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" :: "r"(tmem_base), "r"(TMEM_COLS) : "memory");
    }
}

template <int DQ, int DV, int NB, Weights W>
static int launch(const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv, const Prompt& a, cudaStream_t st) {
    const size_t smem = sizeof(Smem<DQ, NB * DV, W != LAGGING>) + 1024;
    static_assert(sizeof(Smem<DQ, NB * DV, W != LAGGING>) + 1024 <= 227 * 1024 && NB * DV <= 256, "shared and tensor memory of one CTA");
    cudaError_t e = cudaFuncSetAttribute(packed_attn_tc_kernel<DQ, DV, NB, W>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    packed_attn_tc_kernel<DQ, DV, NB, W><<<dim3(a.n, a.H, a.cross ? (a.G + NB - 1) / NB : 1), THREADS, smem, st>>>(mq, mk, mv, a);
    return (int)cudaGetLastError();
}

template <int DQ, Weights W>
static int by_values(const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv, const Prompt& a, cudaStream_t st) {
    const int heads = a.cross ? a.G : 1;
    if (a.dv <= 64)
        return heads > 2   ? launch<DQ, 64, 4, W>(mq, mk, mv, a, st)
               : heads > 1 ? launch<DQ, 64, 2, W>(mq, mk, mv, a, st)
                           : launch<DQ, 64, 1, W>(mq, mk, mv, a, st);
    return heads > 1 ? launch<DQ, 128, 2, W>(mq, mk, mv, a, st) : launch<DQ, 128, 1, W>(mq, mk, mv, a, st);
}

template <int DQ>
static int sigmoid_by_values(const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv, const Prompt& a, cudaStream_t st) {
    return a.dv <= 64    ? launch<DQ, 64, 1, SIGMOID>(mq, mk, mv, a, st)
           : a.dv <= 128 ? launch<DQ, 128, 1, SIGMOID>(mq, mk, mv, a, st)
           : a.dv <= 192 ? launch<DQ, 192, 1, SIGMOID>(mq, mk, mv, a, st)
                         : launch<DQ, 256, 1, SIGMOID>(mq, mk, mv, a, st);
}

}  // namespace patc
}  // namespace lmoe

using namespace lmoe;

// bf16; q [q_rows, ldq], k / v [k_rows, ldk / ldv], gate [q_rows, ldg] or null: bases 16-byte aligned, pitches and head sizes
// multiples of 8, head sizes up to 128 (with sigmoid weights: values up to 256), scale > 0 (sigmoid: of any sign).  items: up to 128 queries each; every row they name lies inside the matrices.
LMOE_API int lmoe_packed_attn_tc(const pa::Prompt* ap, cudaStream_t st) {
    using namespace lmoe::patc;
    const Prompt& a = *ap;
    if (a.n <= 0 || a.q_rows <= 0 || a.k_rows <= 0 || a.H <= 0 || a.G <= 0 || a.H % a.G || a.dk <= 0 || a.dk > 128 || a.dv <= 0 || a.dv > (a.bias != nullptr ? 256 : 128) ||
        a.dk % 8 || a.dv % 8 || a.ldq % 8 || a.ldk % 8 || a.ldv % 8 || a.ldo % 8 || (a.gate != nullptr && a.ldg % 8) ||
        (a.bias == nullptr ? !(a.scale > 0.f) : a.cross || a.gate != nullptr) ||
        (a.cross && a.gate != nullptr) || ((reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(a.k) | reinterpret_cast<uintptr_t>(a.v) |
          reinterpret_cast<uintptr_t>(a.gate) | reinterpret_cast<uintptr_t>(a.out)) & 15))
        return -1;
    CUtensorMap mq, mk, mv;
    int rc = make_map_4d(&mq, a.q, 1, a.q_rows, a.H, a.dk, (long long)a.q_rows * a.ldq, a.ldq, a.dk, BM);
    if (rc == 0) rc = make_map_4d(&mk, a.k, 1, a.k_rows, a.G, a.dk, (long long)a.k_rows * a.ldk, a.ldk, a.dk, BN);
    if (rc == 0) rc = make_map_4d(&mv, a.v, 1, a.k_rows, a.G, a.dv, (long long)a.k_rows * a.ldv, a.ldv, a.dv, 64);
    if (rc) return rc;
    if (a.bias != nullptr) return a.dk <= 64 ? sigmoid_by_values<64>(mq, mk, mv, a, st) : sigmoid_by_values<128>(mq, mk, mv, a, st);
    if (a.cross && a.bounded) return a.dk <= 64 ? by_values<64, BOUNDED_SOFTMAX>(mq, mk, mv, a, st) : by_values<128, BOUNDED_SOFTMAX>(mq, mk, mv, a, st);
    return a.dk <= 64 ? by_values<64, LAGGING>(mq, mk, mv, a, st) : by_values<128, LAGGING>(mq, mk, mv, a, st);
}
