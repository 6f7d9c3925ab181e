// Chunked, soft-capped, distance-biased, gated attention over prompts on the 5th-generation tensor cores (bf16, head sizes up
// to 128 in multiples of 8).  The mathematics and the operand layout are those of chunk_attn.cu.
//
// A soft cap bounds every score by cap + max|bias|, so exp(score) cannot leave fp32 (the host takes this kernel only while that
// bound is at most 60) and the softmax needs no running maximum: P = exp(S) as it is, O accumulates in tensor memory over all
// key tiles, and only the row sums are added up at the end.  No rescaling, no exchange between the threads of a row.
//
// One CTA = up to 128 queries of one head inside one chunk (work items, longest first).  Warp roles as in flash_attn_tc.cu:
//   warp 0      TMA producer: Q once, then K_j / V_j tiles of 128 keys through two 2-stage rings; head sizes below 64 / 128 are
//               filled up with zeros by the tensor map's bounds
//   warp 1      MMA issuer: S_{j+1} = Q K_{j+1}^T before O += P_j V_j
//   warps 4..19 four warps per 32 query rows split the columns: one tensor-memory read of the scores,
//                   e = 2^(2 s scale log2(e) / cap),  tanh = 1 - 2 / (e + 1),  P = 2^(cap' tanh + bias')
//               (three special-function operations and one shared-memory read per score; primes: in units of log2), bf16 pack into
//               the 128-byte-swizzled P tile, row sums in registers
// The bias table of the head sits in shared memory, shifted and padded so that a tile needs no clamping of its index; tiles
// entirely beyond the table's end use its last value.
// Every mbarrier wait is bounded; on expiry the error word is set and the CTA drains and frees its tensor memory.
#include "attn_math.cuh"
#include "chunk_attn.cuh"
#include "flash_tc_utils.cuh"

namespace lmoe {
namespace catc {
using namespace lmoe::fatc;

constexpr int LUT_NEG = 256, LUT_TAIL = 256, LUT_MAX = 4096;          // table floats: 256 before distance 0 and behind the end

struct Args {
    const int* items;         // [n, 8]
    const bf16* gate;         // column zg of the projection output
    bf16* out;
    const float* lut;         // [H, nlut]
    const float* gain;
    int* err;
    long long ldz, ldo;
    int nlut, H, G, dv;
    float scale, cap, mul;
};

template <int DQ, int DV>
struct __align__(1024) Smem {
    uint8_t q[BM * DQ * 2];
    uint8_t k[2][BN * DQ * 2];
    uint8_t v[2][BN * DV * 2];
    uint8_t p[BM * BN * 2];
    float lut[LUT_MAX];
    float ls[SPLIT][BM];
    uint64_t q_full, k_full[2], k_empty[2], v_full[2], v_empty[2], s_full[2], pv_done, p_ready;
    uint32_t tmem_base;
    int abort_flag;
};

template <int DQ, int DV>
__global__ void __launch_bounds__(THREADS, 1)
chunk_attn_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                     const __grid_constant__ CUtensorMap tmV, Args a) {
    extern __shared__ uint8_t smem_raw[];
    Smem<DQ, DV>& sm = *reinterpret_cast<Smem<DQ, DV>*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    constexpr int KQ = DQ / 64, KV = DV / 64;               // 64-element blocks along the head dimensions
    constexpr uint32_t TMEM_COLS = 512, O_COL = 2 * BN;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int* it = a.items + (long long)blockIdx.x * I_N;
    const int row0 = it[I_ROW], nq = it[I_NQ], c0 = it[I_C0];
    const int h = blockIdx.y, hk = h / (a.H / a.G);
    const int n_it = (c0 + nq + BN - 1) / BN;               // at least 1
    volatile int* abort_flag = &sm.abort_flag;
    int* err = a.err;

    if (threadIdx.x == 0) {
        mbar_init(&sm.q_full, 1);
        for (int s = 0; s < 2; ++s) {
            mbar_init(&sm.k_full[s], 1); mbar_init(&sm.k_empty[s], 1);
            mbar_init(&sm.v_full[s], 1); mbar_init(&sm.v_empty[s], 1);
            mbar_init(&sm.s_full[s], 1);
        }
        mbar_init(&sm.pv_done, 1);
        mbar_init(&sm.p_ready, 4 * SPLIT);
        sm.abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" :: "r"(s32(&sm.tmem_base)), "r"(TMEM_COLS) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    // lut[LUT_NEG + d] = bias(d) log2(e) + cap log2(e) for the distances this item can see
    const float cap2 = a.cap * LOG2E;
    {
        const int used = LUT_NEG + min(a.nlut, c0 + nq) + LUT_TAIL;
        const float* src = a.lut + (long long)h * a.nlut;
        for (int i = threadIdx.x; i < used; i += THREADS) sm.lut[i] = src[min(max(i - LUT_NEG, 0), a.nlut - 1)] * LOG2E + cap2;
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
                const int key0 = row0 - c0 + j * BN;        // packed row of the tile's first key
                if (!mbar_wait_suspend(&sm.k_empty[s], ph ^ 1, abort_flag, err, 0x4100 | s)) break;
                mbar_expect_tx(&sm.k_full[s], BN * DQ * 2);
#pragma unroll
                for (int kb = 0; kb < KQ; ++kb) tma_load_4d(sm.k[s] + kb * BN * 128, &tmK, &sm.k_full[s], kb * 64, hk, key0, 0);
                if (!mbar_wait_suspend(&sm.v_empty[s], ph ^ 1, abort_flag, err, 0x4200 | s)) break;
                mbar_expect_tx(&sm.v_full[s], BN * DV * 2);
#pragma unroll
                for (int kk = 0; kk < BN / 64; ++kk)        // MN-major operand: per 64 keys, DV/64 boxes of {64 d, 64 keys}
#pragma unroll
                    for (int nb = 0; nb < KV; ++nb)
                        tma_load_4d(sm.v[s] + (kk * KV + nb) * 8192, &tmV, &sm.v_full[s], nb * 64, hk, key0 + kk * 64, 0);
            }
        }
    } else if (warp == 1) {
        const uint32_t issue = lane == 0 ? 1u : 0u;
        constexpr uint32_t idesc_s = idesc_bf16<false, BN>();
        constexpr uint32_t idesc_o = idesc_bf16<true, DV>();
        bool ok = mbar_wait_suspend(&sm.q_full, 0, abort_flag, err, 0x5000);
        auto issue_s = [&](int j) -> bool {
            const int s = j & 1;
            if (!mbar_wait_suspend(&sm.k_full[s], (j >> 1) & 1, abort_flag, err, 0x5100 | s)) return false;
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
            // score buffer (j + 1) & 1 was last read for P_{j-1}, whose p_ready was waited for in the previous iteration
            if (j + 1 < n_it) { ok = issue_s(j + 1); if (!ok) break; }
            const int s = j & 1;
            if (!mbar_wait_suspend(&sm.v_full[s], (j >> 1) & 1, abort_flag, err, 0x5200 | s)) break;
            if (!mbar_wait_suspend(&sm.p_ready, j & 1, abort_flag, err, 0x5300)) break;
            tc_fence_after();
            const uint32_t pl = desc_lo<false>(s32(sm.p)), vl = desc_lo<true>(s32(sm.v[s]));
#pragma unroll
            for (int kk = 0; kk < BN / UMMA_K; ++kk) {
                const uint32_t aoff = ((kk / 4) * (BM * 128) + (kk % 4) * 32) >> 4;
                const uint32_t boff = ((kk / 4) * (KV * 8192) + (kk % 4) * 2048) >> 4;
                umma_lo(tmem_base + O_COL, pl + aoff, vl + boff, idesc_o, (j > 0 || kk > 0) ? 1u : 0u, issue);
            }
            umma_commit_if(&sm.v_empty[s], issue);
            umma_commit_if(&sm.pv_done, issue);
        }
    } else if (warp >= 4) {
        const int qd = warp & 3, part = (warp - 4) >> 2;
        const int r = qd * 32 + lane;                         // query row inside the tile
        const uint32_t lane_addr = tmem_base + ((uint32_t)(qd * 32) << 16);
        constexpr int CW = BN / SPLIT, OW = DV / SPLIT;       // score / output columns of this thread
        static_assert(CW == 32, "one 32-column tensor-memory load per tile");
        const float gain = *a.gain;
        const float k1 = 2.f * LOG2E * a.scale * gain * gain / a.cap, m2 = -2.f * cap2;
        uint8_t* prow = sm.p + ((part * CW) >> 6) * (BM * 128) + (r >> 3) * 1024 + (r & 7) * 128;
        const int ch0 = ((part * CW) & 63) >> 3;
        float ps[4] = {0.f, 0.f, 0.f, 0.f};
        bool alive = true;
        for (int j = 0; j < n_it; ++j) {
            const int s = j & 1, tile0 = j * BN;
            const int dist0 = c0 + r - (tile0 + part * CW);    // distance of this thread's first column
            if (!mbar_wait_suspend(&sm.s_full[s], (j >> 1) & 1, abort_flag, err, 0x6100 | s)) { alive = false; break; }
            tc_fence_after();
            uint32_t v[CW];
            tmem_ld32(lane_addr + s * BN + part * CW, v);
            tmem_ld_wait();
            const bool far = c0 - (tile0 + BN - 1) >= a.nlut - 1;      // the whole tile has the table's last value
            const bool diag = tile0 + BN - 1 > c0;
            const float* lp = far ? &sm.lut[LUT_NEG + a.nlut - 1] : &sm.lut[LUT_NEG + dist0];
            auto weight = [&](float x, float b2) {
                const float e = ex2(x * k1);
                return ex2(fmaf(rcp(e + 1.f), m2, b2));
            };
            if (far) {
                const float b2 = lp[0];
#pragma unroll
                for (int c = 0; c < CW; ++c) v[c] = __float_as_uint(weight(__uint_as_float(v[c]), b2));
            } else {
#pragma unroll
                for (int c = 0; c < CW; ++c) v[c] = __float_as_uint(weight(__uint_as_float(v[c]), lp[-c]));
            }
            if (diag) {
#pragma unroll
                for (int c = 0; c < CW; ++c)
                    if (c > dist0) v[c] = 0u;
            }
#pragma unroll
            for (int c = 0; c < CW; c += 4) {
#pragma unroll
                for (int e = 0; e < 4; ++e) ps[e] += __uint_as_float(v[c + e]);
                v[c >> 1] = pack_bf16(__uint_as_float(v[c]), __uint_as_float(v[c + 1]));
                v[(c >> 1) + 1] = pack_bf16(__uint_as_float(v[c + 2]), __uint_as_float(v[c + 3]));
            }
            // the P tile is free once O += P_{j-1} V_{j-1} has completed
            if (j > 0 && !mbar_wait_suspend(&sm.pv_done, (j - 1) & 1, abort_flag, err, 0x6200)) { alive = false; break; }
#pragma unroll
            for (int c = 0; c < 4; ++c)
                *reinterpret_cast<uint4*>(prow + (((ch0 + c) ^ (r & 7)) << 4)) = make_uint4(v[4 * c], v[4 * c + 1], v[4 * c + 2], v[4 * c + 3]);
            tc_fence_before();
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(&sm.p_ready);
        }
        if (alive) alive = mbar_wait_suspend(&sm.pv_done, (n_it - 1) & 1, abort_flag, err, 0x6300);
        tc_fence_after();
        sm.ls[part][r] = (ps[0] + ps[1]) + (ps[2] + ps[3]);
        asm volatile("bar.sync %0, %1;" :: "r"(1 + qd), "n"(32 * SPLIT) : "memory");
        float l = 0.f;
#pragma unroll
        for (int p = 0; p < SPLIT; ++p) l += sm.ls[p][r];
        uint32_t o[OW];
        tmem_ld<OW>(lane_addr + O_COL + part * OW, o);
        tmem_ld_wait();
        if (alive && r < nq) {
            const float w = a.mul * gain / l;
            const long long row = row0 + r;
            const bf16* gp = a.gate + row * a.ldz + h * a.dv;
            bf16* op = a.out + row * a.ldo + h * a.dv;
#pragma unroll
            for (int c = 0; c < OW; c += 8) {
                const int col = part * OW + c;
                if (col < a.dv) {
                    Vec<bf16> g, y;
                    g.load(gp + col);
#pragma unroll
                    for (int i = 0; i < 8; ++i)
                        y.set(i, __uint_as_float(o[c + i]) * w * rcp(1.f + ex2(-LOG2E * gain * g.get(i))));
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

template <int DQ, int DV>
static int launch(const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv, const Args& a, int n, cudaStream_t st) {
    const size_t smem = sizeof(Smem<DQ, DV>) + 1024;
    static_assert(sizeof(Smem<DQ, DV>) + 1024 <= 227 * 1024, "shared memory of one CTA");
    cudaError_t e = cudaFuncSetAttribute(chunk_attn_tc_kernel<DQ, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    chunk_attn_tc_kernel<DQ, DV><<<dim3(n, a.H), THREADS, smem, st>>>(mq, mk, mv, a);
    return (int)cudaGetLastError();
}

}  // namespace catc
}  // namespace lmoe

using namespace lmoe;

// z [rows, ldz] bf16 with queries, keys, values, gates from columns zq, zk, zv, zg (multiples of 8, as are dk, dv, ldz, ldo; 16-byte
// aligned bases).  items [n, 8]: as for lmoe_chunk_attn_rows, with up to 128 queries, and every key of the chunk in this call.
LMOE_API int lmoe_chunk_attn_tc(const bf16* z, int rows, int zq, int zk, int zv, int zg, int dk, const catc::Args* ap, int n,
                                cudaStream_t st) {
    using namespace lmoe::catc;
    Args a = *ap;
    if (n <= 0 || rows <= 0 || dk <= 0 || dk > 128 || a.dv <= 0 || a.dv > 128 || dk % 8 || a.dv % 8 || a.ldz % 8 || a.ldo % 8 || a.H % a.G ||
        ((zq | zk | zv | zg) & 7) || (reinterpret_cast<uintptr_t>(z) & 15) || (reinterpret_cast<uintptr_t>(a.out) & 15) || !(a.cap > 0.f) ||
        a.nlut <= 0 || a.nlut + LUT_NEG + LUT_TAIL > LUT_MAX)
        return -1;
    a.gate = z + zg;
    CUtensorMap mq, mk, mv;
    const long long sb = (long long)rows * a.ldz;
    int rc = make_map_4d(&mq, z + zq, 1, rows, a.H, dk, sb, a.ldz, dk, BM);
    if (rc == 0) rc = make_map_4d(&mk, z + zk, 1, rows, a.G, dk, sb, a.ldz, dk, BN);
    if (rc == 0) rc = make_map_4d(&mv, z + zv, 1, rows, a.G, a.dv, sb, a.ldz, a.dv, 64);
    if (rc) return rc;
    if (dk <= 64) return a.dv <= 64 ? launch<64, 64>(mq, mk, mv, a, n, st) : launch<64, 128>(mq, mk, mv, a, n, st);
    return a.dv <= 64 ? launch<128, 64>(mq, mk, mv, a, n, st) : launch<128, 128>(mq, mk, mv, a, n, st);
}
