// Building blocks of the tcgen05 attention kernels (flash_attn_tc.cu, chunk_attn_tc.cu): 4-D TMA loads over [B, T, H, D],
// tensor-memory reads, MMA issue by a converged warp, bounded suspending mbarrier waits and the tensor-map encoder.
#pragma once
#include <cstdio>
#include "tcgen05_utils.cuh"

namespace lmoe {
namespace fatc {
using namespace lmoe::tc;

constexpr int BM = 128, BN = 128, SPLIT = 4, THREADS = 128 + 128 * SPLIT, UMMA_K = 16;
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ void tma_load_4d(void* dst, const CUtensorMap* map, uint64_t* bar, int c0, int c1, int c2, int c3) {
    asm volatile("cp.async.bulk.tensor.4d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5, %6}], [%2];"
                 :: "r"(s32(dst)), "l"(map), "r"(s32(bar)), "r"(c0), "r"(c1), "r"(c2), "r"(c3) : "memory");
}
template <bool B_MN, int N>
__host__ __device__ constexpr uint32_t idesc_bf16() {
    return (1u << 4) | (1u << 7) | (1u << 10) | ((B_MN ? 1u : 0u) << 16) | ((uint32_t)(N >> 3) << 17) | ((uint32_t)(BM >> 4) << 24);
}

__device__ __forceinline__ void tmem_ld64(uint32_t taddr, uint32_t (&r)[64]) {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x64.b32 "
                 "{%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31,"
                 "%32,%33,%34,%35,%36,%37,%38,%39,%40,%41,%42,%43,%44,%45,%46,%47,%48,%49,%50,%51,%52,%53,%54,%55,%56,%57,%58,%59,%60,%61,%62,%63}, [%64];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]),
                   "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]),
                   "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]),
                   "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31]),
                   "=r"(r[32]), "=r"(r[33]), "=r"(r[34]), "=r"(r[35]), "=r"(r[36]), "=r"(r[37]), "=r"(r[38]), "=r"(r[39]),
                   "=r"(r[40]), "=r"(r[41]), "=r"(r[42]), "=r"(r[43]), "=r"(r[44]), "=r"(r[45]), "=r"(r[46]), "=r"(r[47]),
                   "=r"(r[48]), "=r"(r[49]), "=r"(r[50]), "=r"(r[51]), "=r"(r[52]), "=r"(r[53]), "=r"(r[54]), "=r"(r[55]),
                   "=r"(r[56]), "=r"(r[57]), "=r"(r[58]), "=r"(r[59]), "=r"(r[60]), "=r"(r[61]), "=r"(r[62]), "=r"(r[63])
                 : "r"(taddr));
}
__device__ __forceinline__ void tmem_ld16(uint32_t taddr, uint32_t (&r)[16]) {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]),
                   "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
                 : "r"(taddr));
}
template <int N>
__device__ __forceinline__ void tmem_ld(uint32_t taddr, uint32_t (&r)[N]) {
    static_assert(N == 16 || N == 32 || N == 64, "tensor-memory load width");
    if constexpr (N == 64) tmem_ld64(taddr, r);
    else if constexpr (N == 32) tmem_ld32(taddr, r);
    else tmem_ld16(taddr, r);
}
// o[i] = o[i] * corr + partial[i] for this thread's OW columns of the partial output in tensor memory
template <int OW>
__device__ __forceinline__ void fold_o(float (&o)[OW], uint32_t taddr, float corr) {
    uint32_t v[OW];
    tmem_ld<OW>(taddr, v);
    tmem_ld_wait();
    const float2 c2 = make_float2(corr, corr);
#pragma unroll
    for (int i = 0; i < OW; i += 2) {                            // packed fp32 FMAs: two columns per instruction
        const float2 r = __ffma2_rn(make_float2(o[i], o[i + 1]), c2, make_float2(__uint_as_float(v[i]), __uint_as_float(v[i + 1])));
        o[i] = r.x;
        o[i + 1] = r.y;
    }
}
// The MMA warp runs its loop with all 32 lanes converged and only predicates the tcgen05 instructions on one lane: inside a
// single-lane branch every operand lives in vector registers and each MMA pays for moving two 64-bit descriptors into
// uniform registers, which at 64-column tiles costs more cycles than the MMA keeps the tensor core busy.  Descriptors are
// built once per tile as a 32-bit low word (address / 16 and the leading-dimension offset); the high word is a constant and
// stepping along K inside the swizzled tile is an add to the low word.
constexpr uint32_t DESC_HI = (1024u >> 4) | (1u << 14) | (2u << 29);      // stride offset 1024 B, version 1, 128-byte swizzle
template <bool MN>
__device__ __forceinline__ uint32_t desc_lo(uint32_t saddr) {
    return ((saddr >> 4) & 0x3FFFu) | ((MN ? (8192u >> 4) : 1u) << 16);
}
__device__ __forceinline__ void umma_lo(uint32_t tmem_d, uint32_t a_lo, uint32_t b_lo, uint32_t idesc, uint32_t accumulate, uint32_t issue) {
    asm volatile("{\n.reg .pred p, q;\n.reg .b64 da, db;\nsetp.ne.b32 p, %4, 0;\nsetp.ne.b32 q, %5, 0;\n"
                 "mov.b64 da, {%1, %6};\nmov.b64 db, {%2, %6};\n"
                 "@q tcgen05.mma.cta_group::1.kind::f16 [%0], da, db, %3, p;\n}"
                 :: "r"(tmem_d), "r"(a_lo), "r"(b_lo), "r"(idesc), "r"(accumulate), "r"(issue), "r"(DESC_HI) : "memory");
}
__device__ __forceinline__ void umma_commit_if(uint64_t* bar, uint32_t issue) {
    asm volatile("{\n.reg .pred q;\nsetp.ne.b32 q, %1, 0;\n"
                 "@q tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];\n}" :: "r"(s32(bar)), "r"(issue) : "memory");
}
__device__ __forceinline__ float max3(float a, float b, float c) {
    float r;
    asm("max.f32 %0, %1, %2, %3;" : "=f"(r) : "f"(a), "f"(b), "f"(c));
    return r;
}
// Bounded wait that lets the hardware suspend the warp (try_wait with a time hint) instead of spinning on test_wait:
// the 16 softmax warps share 4 schedulers, a spinning warp takes issue slots from the others.
__device__ __forceinline__ bool mbar_try_suspend(uint64_t* bar, uint32_t parity) {
    uint32_t ok;
    asm volatile("{\n.reg .pred p;\nmbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2, %3;\nselp.u32 %0, 1, 0, p;\n}"
                 : "=r"(ok) : "r"(s32(bar)), "r"(parity), "r"(20000u) : "memory");
    return ok != 0;
}
__device__ __forceinline__ bool mbar_wait_suspend(uint64_t* bar, uint32_t parity, volatile int* abort_flag, int* err, int code) {
    if (mbar_try_suspend(bar, parity)) return true;
    const long long t0 = clock64();
    for (;;) {
        if (mbar_try_suspend(bar, parity)) return true;
        if (*abort_flag) return false;
        if (clock64() - t0 > WAIT_CYCLES) break;
    }
    *abort_flag = 1;
    atomicCAS(err, 0, code);
    return false;
}

// [B, T, H, D] bf16 with element strides (sb, st, sh), unit stride along D; box = {64, 1, box_t, 1}
static int make_map_4d(CUtensorMap* map, const void* ptr, int B, int T, int H, int D, long long sb, long long st, long long sh,
                       uint32_t box_t) {
    EncodeTiledFn enc = get_encode();
    if (enc == nullptr) return -10;
    cuuint64_t dims[4] = {(cuuint64_t)D, (cuuint64_t)H, (cuuint64_t)T, (cuuint64_t)B};
    cuuint64_t strides[3] = {(cuuint64_t)sh * 2, (cuuint64_t)st * 2, (cuuint64_t)sb * 2};
    cuuint32_t box[4] = {64, 1, box_t, 1};
    cuuint32_t estr[4] = {1, 1, 1, 1};
    CUresult r = enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, const_cast<void*>(ptr), dims, strides, box, estr,
                     CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                     CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS)
        fprintf(stderr, "flash_attn_tc: tensor map rejected (CUresult %d): ptr %p dims {%d,%d,%d,%d} strides {%lld,%lld,%lld} box_t %u\n",
                (int)r, ptr, D, H, T, B, sh, st, sb, box_t);
    return r == CUDA_SUCCESS ? 0 : -11;
}

}  // namespace fatc
}  // namespace lmoe
