// One-token step of chunked, soft-capped, distance-biased, gated attention for bf16 (mathematics, arguments and cache layout:
// chunk_attn.cu), bound by reading the request's cached keys and values once.
//
// A warp works on 16 keys at a time, straight from global memory into mma.sync fragments; nothing is staged:
//   S^T [16 keys x 8 heads] = K Q^T    the 8 consecutive dims that a lane loads (16 bytes) are the k slots it owns in two MMA steps;
//                                      the sum does not care about the order as long as K and Q agree
//   P = exp(S)                         as in chunk_attn_tc.cu the soft cap bounds the scores (checked on the host): no maximum, so
//                                      warps, CTAs and iterations only add up
//   O^T [dims x 8 heads] += V^T P^T    a lane loads 8 dims of the four keys whose k slots it owns; byte permutes pair the keys, and
//                                      the 8x8 transposes of P are movmatrix instructions
// The keys of (request, kv head) are split over the warps of a CTA and the CTAs of a cluster; partial sums meet in (distributed)
// shared memory, where the gate is applied.  The new token's key and value come from the projection and are stored into the cache.
// While the kernel before it (the projection) still runs, it fetches the first cached keys and values.
#include <cooperative_groups.h>

#include "attn_math.cuh"
#include "chunk_attn.cuh"
#include "common.cuh"
#include "mma_utils.cuh"

namespace lmoe {
namespace cas {
namespace cg = cooperative_groups;

constexpr int WARPS = 4, HEADS = 8;
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ uint32_t pack2(float lo, float hi) {
    __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&h);
}
__device__ __forceinline__ uint32_t transpose8x8(uint32_t x) {
    uint32_t r;
    asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(r) : "r"(x));
    return r;
}
__device__ __forceinline__ uint32_t word(const uint4& v, int i) { return i == 0 ? v.x : i == 1 ? v.y : i == 2 ? v.z : v.w; }

// KG: groups of 32 key dims, VG: groups of 64 value dims.  grid (splits, G * head tiles, B), cluster (splits, 1, 1)
template <int KG, int VG>
__global__ void __launch_bounds__(WARPS * 32) chunk_attn_step_mma_kernel(ca::Args a) {
    constexpr int DV = VG * 64;
    __shared__ float part[WARPS][HEADS][DV + 1];             // [warp][head][dim], last column: row sum
    __shared__ float sum[HEADS][DV + 1];
    const int w = threadIdx.x >> 5, l = threadIdx.x & 31, g = l >> 2, q = l & 3;
    const int splits = gridDim.x, split = blockIdx.x, b = blockIdx.z;
    const int qpg = a.H / a.G, tiles = (qpg + HEADS - 1) / HEADS;
    const int hk = blockIdx.y / tiles, h0 = hk * qpg + (blockIdx.y % tiles) * HEADS;
    const int nh = min(HEADS, hk * qpg + qpg - h0);
    const int slot = a.slots[b], cur = a.pos[b] % a.size, nk = cur + 1;
    constexpr int STEP = 16 * WARPS;
    const int per = ((nk + splits - 1) / splits + STEP - 1) / STEP * STEP;
    const int k_lo = split * per, k_hi = min(nk, k_lo + per);
    const bf16* zrow = (const bf16*)a.z + (long long)b * a.ldz;
    const bf16* kc = (const bf16*)a.kc + ((long long)slot * a.cap_rows * a.G + hk) * a.dkp;
    const bf16* vc = (const bf16*)a.vc + ((long long)slot * a.cap_rows * a.G + hk) * a.dvp;
    const long long k_pitch = (long long)a.G * a.dkp, v_pitch = (long long)a.G * a.dvp;
    const uint4 zero = make_uint4(0, 0, 0, 0);

    auto load_k = [&](uint4 (&kf)[2][KG], int key0, bool all) {        // all: also the new token (its row of z is complete)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int key = key0 + g + 8 * r;
            const bf16* p = key == cur ? zrow + a.zk + hk * a.dk : kc + key * k_pitch;
            const bool ok = key < k_hi && (all || key != cur);
#pragma unroll
            for (int i = 0; i < KG; ++i) {
                const int d = i * 32 + q * 8;
                kf[r][i] = ok && d < a.dk ? __ldcs(reinterpret_cast<const uint4*>(p + d)) : zero;
            }
        }
    };
    auto load_v = [&](uint4 (&vf)[4][VG], int key0, bool all) {
#pragma unroll
        for (int r = 0; r < 4; ++r) {
            const int key = key0 + 2 * q + (r & 1) + 8 * (r >> 1);
            const bf16* p = key == cur ? zrow + a.zv + hk * a.dv : vc + key * v_pitch;
            const bool ok = key < k_hi && (all || key != cur);
#pragma unroll
            for (int i = 0; i < VG; ++i) {
                const int d = i * 64 + g * 8;
                vf[r][i] = ok && d < a.dv ? __ldcs(reinterpret_cast<const uint4*>(p + d)) : zero;
            }
        }
    };

    uint4 kf[2][KG], vf[4][VG];
    int key0 = k_lo + 16 * w;
    const bool holds_cur = cur >= key0 && cur < key0 + 16;             // then the first tile has to wait for the projection
    if (!holds_cur) {
        load_k(kf, key0, false);
        load_v(vf, key0, false);
    }
    pdl_trigger();
    asm volatile("griddepcontrol.wait;" ::: "memory");
    if (holds_cur) {
        load_k(kf, key0, true);
        load_v(vf, key0, true);
    }
    const float gain = *a.gain;
    uint4 qf[KG];                                                      // head h0 + g
#pragma unroll
    for (int i = 0; i < KG; ++i) {
        const int d = i * 32 + q * 8;
        qf[i] = g < nh && d < a.dk ? *reinterpret_cast<const uint4*>(zrow + a.zq + (h0 + g) * a.dk + d) : zero;
    }
    // the new key and value enter the cache
    if (h0 == hk * qpg && cur >= k_lo && cur < k_hi) {
        bf16* kd = (bf16*)a.kc + (((long long)slot * a.cap_rows + cur) * a.G + hk) * a.dkp;
        bf16* vd = (bf16*)a.vc + (((long long)slot * a.cap_rows + cur) * a.G + hk) * a.dvp;
        for (int d = threadIdx.x * 8; d < a.dk; d += WARPS * 256)
            *reinterpret_cast<uint4*>(kd + d) = *reinterpret_cast<const uint4*>(zrow + a.zk + hk * a.dk + d);
        for (int d = threadIdx.x * 8; d < a.dv; d += WARPS * 256)
            *reinterpret_cast<uint4*>(vd + d) = *reinterpret_cast<const uint4*>(zrow + a.zv + hk * a.dv + d);
    }
    const float cap2 = a.cap * LOG2E, k1 = 2.f * LOG2E * a.scale * gain * gain / a.cap;
    // this lane's scores belong to heads 2q, 2q + 1 of the tile
    const bool on0 = 2 * q < nh, on1 = 2 * q + 1 < nh;
    const float* lut0 = a.lut + (long long)(h0 + (on0 ? 2 * q : 0)) * a.nlut;
    const float* lut1 = a.lut + (long long)(h0 + (on1 ? 2 * q + 1 : 0)) * a.nlut;
    auto weight = [&](float s, float bias) { return ex2(fmaf(-2.f * cap2, rcp(ex2(s * k1) + 1.f), fmaf(bias, LOG2E, cap2))); };
    float o[VG * 4][4];
#pragma unroll
    for (int t = 0; t < VG * 4; ++t) o[t][0] = o[t][1] = o[t][2] = o[t][3] = 0.f;
    float l0 = 0.f, l1 = 0.f;
    for (; key0 < k_hi; key0 += STEP) {
        float s[4] = {0.f, 0.f, 0.f, 0.f};                             // (key g, key g + 8) x (head 2q, head 2q + 1)
#pragma unroll
        for (int i = 0; i < KG; ++i) {
            const uint32_t f1[4] = {kf[0][i].x, kf[1][i].x, kf[0][i].y, kf[1][i].y};
            const uint32_t f2[4] = {kf[0][i].z, kf[1][i].z, kf[0][i].w, kf[1][i].w};
            mma16816(s, f1, qf[i].x, qf[i].y);
            mma16816(s, f2, qf[i].z, qf[i].w);
        }
        if (key0 + STEP < k_hi) load_k(kf, key0 + STEP, true);
        const int d0 = cur - (key0 + g), d1 = d0 - 8;                  // distances; negative past the end
        const int i0 = min(max(d0, 0), a.nlut - 1), i1 = min(max(d1, 0), a.nlut - 1);
        const bool v0 = key0 + g < k_hi, v1 = key0 + g + 8 < k_hi;
        const float p00 = v0 && on0 ? weight(s[0], lut0[i0]) : 0.f, p01 = v0 && on1 ? weight(s[1], lut1[i0]) : 0.f;
        const float p10 = v1 && on0 ? weight(s[2], lut0[i1]) : 0.f, p11 = v1 && on1 ? weight(s[3], lut1[i1]) : 0.f;
        l0 += p00 + p10;
        l1 += p01 + p11;
        const uint32_t b0 = transpose8x8(pack2(p00, p01)), b1 = transpose8x8(pack2(p10, p11));
#pragma unroll
        for (int i = 0; i < VG; ++i)
#pragma unroll
            for (int t = 0; t < 4; ++t) {                              // rows g, g + 8 of the tile: dims 2t, 2t + 1 of this lane's eight
                const uint32_t w0 = word(vf[0][i], t), w1 = word(vf[1][i], t), w2 = word(vf[2][i], t), w3 = word(vf[3][i], t);
                const uint32_t f[4] = {__byte_perm(w0, w1, 0x5410), __byte_perm(w0, w1, 0x7632), __byte_perm(w2, w3, 0x5410),
                                       __byte_perm(w2, w3, 0x7632)};
                mma16816(o[i * 4 + t], f, b0, b1);
            }
        if (key0 + STEP < k_hi) load_v(vf, key0 + STEP, true);
    }
#pragma unroll
    for (int x = 4; x < 32; x <<= 1) {                                 // over the lanes with the same q
        l0 += __shfl_xor_sync(0xffffffffu, l0, x);
        l1 += __shfl_xor_sync(0xffffffffu, l1, x);
    }
#pragma unroll
    for (int i = 0; i < VG; ++i)
#pragma unroll
        for (int t = 0; t < 4; ++t) {
            const int d = i * 64 + g * 8 + 2 * t;
            part[w][2 * q][d] = o[i * 4 + t][0];
            part[w][2 * q + 1][d] = o[i * 4 + t][1];
            part[w][2 * q][d + 1] = o[i * 4 + t][2];
            part[w][2 * q + 1][d + 1] = o[i * 4 + t][3];
        }
    if (g == 0) {
        part[w][2 * q][DV] = l0;
        part[w][2 * q + 1][DV] = l1;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < HEADS * (DV + 1); i += WARPS * 32) {
        float v = 0.f;
#pragma unroll
        for (int k = 0; k < WARPS; ++k) v += (&part[k][0][0])[i];
        (&sum[0][0])[i] = v;
    }
    auto cluster = cg::this_cluster();
    cluster.sync();
    // every CTA of the cluster finishes a slice of the (head, dim) pairs
    for (int i = split * WARPS * 32 + threadIdx.x; i < nh * a.dv; i += splits * WARPS * 32) {
        const int h = i / a.dv, d = i % a.dv;
        float ls = 0.f, os = 0.f;
        for (int r = 0; r < splits; ++r) {
            const float* src = cluster.map_shared_rank(&sum[0][0], r) + h * (DV + 1);
            ls += src[DV];
            os += src[d];
        }
        const int col = (h0 + h) * a.dv + d;
        const float gate = rcp(1.f + ex2(-LOG2E * gain * __bfloat162float(zrow[a.zg + col])));
        ((bf16*)a.out)[(long long)b * a.ldo + col] = __float2bfloat16(os / ls * (a.mul * gain) * gate);
    }
    cluster.sync();                                                    // nobody leaves while its shared memory is read
}

template <int KG, int VG>
static int launch(const ca::Args& a, int splits, cudaStream_t st) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(splits, a.G * ((a.H / a.G + HEADS - 1) / HEADS), a.n);
    cfg.blockDim = dim3(WARPS * 32);
    cfg.stream = st;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = splits;
    attr[0].val.clusterDim.y = 1;
    attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 2;
    return (int)cudaLaunchKernelEx(&cfg, chunk_attn_step_mma_kernel<KG, VG>, a);
}

}  // namespace cas
}  // namespace lmoe

using namespace lmoe;

// As lmoe_chunk_attn_step for bf16, head sizes in multiples of 8 up to 128, a.cap > 0 and scores bounded (|s| <= 60): slots and
// positions must have been on the device before the kernel that precedes this one in the stream was launched.
LMOE_API int lmoe_chunk_attn_step_mma(const ca::Args* ap, int splits, cudaStream_t st) {
    const ca::Args& a = *ap;
    if (a.n <= 0 || a.G <= 0 || a.H % a.G || a.dk <= 0 || a.dv <= 0 || a.dk > 128 || a.dv > 128 || a.dk % 8 || a.dv % 8 || a.dkp % 8 ||
        a.dvp % 8 || a.ldz % 8 || ((a.zq | a.zk | a.zv) & 7) || !(a.cap > 0.f) || a.nlut <= 0 || a.size <= 0 ||
        ((reinterpret_cast<uintptr_t>(a.z) | reinterpret_cast<uintptr_t>(a.kc) | reinterpret_cast<uintptr_t>(a.vc)) & 15) ||
        (splits != 1 && splits != 2 && splits != 4 && splits != 8))
        return -1;
    if (a.dk <= 64) return a.dv <= 64 ? cas::launch<2, 1>(a, splits, st) : cas::launch<2, 2>(a, splits, st);
    return a.dv <= 64 ? cas::launch<4, 1>(a, splits, st) : cas::launch<4, 2>(a, splits, st);
}
