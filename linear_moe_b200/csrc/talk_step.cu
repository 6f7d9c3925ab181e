// One-token attention with talking heads for bf16: the softmax weights of all heads are mixed by a table before they meet the values,
//     o_h = sum over j of (sum over g of T[h, g] softmax_g(j)) v_j            v of h's kv head
// Every output needs the weights of all heads, so a step is two kernels, each of which reads its half of the cache once:
//   talk_scores_kernel   scores of all heads in units of log2 to memory, and every CTA's maximum and sum
//   talk_values_kernel   T / sum as coefficients; the exponentials of 16 keys and all heads times the coefficients on the tensor core
//                        (tf32 in two parts each: fp32 to within its rounding), then the values
// Both work on keys as the one-token kernel of chunk_attn_step.cu does: a warp takes 16 keys straight from global memory into mma.sync
// fragments, the keys of (request, kv head, 8 heads) are split over the warps of a CTA and over CTAs.  Arguments and cache addressing:
// packed_attn.cuh; the new token's key and value are in the cache already.
#include <cooperative_groups.h>

#include "attn_math.cuh"
#include "common.cuh"
#include "mma_utils.cuh"
#include "packed_attn.cuh"

namespace lmoe {
namespace ts {
namespace cg = cooperative_groups;

constexpr int WARPS = 4, HEADS = 8, STEP = 16 * WARPS;
constexpr float LOG2E = 1.4426950408889634f;

struct Args {
    pa::Step s;
    const float* table;                  // [H, H]
    float* scores;                       // [n, H, lds] log2 units, by place of the key in the request's cache
    float* parts;                        // [n, H, splits, 2] maximum and sum of every CTA's keys
    long long lds;
};

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
__device__ __forceinline__ uint32_t tf32(float x) {
    uint32_t r;
    asm("cvt.rna.tf32.f32 %0, %1;" : "=r"(r) : "f"(x));
    return r;
}
__device__ __forceinline__ void mma1688(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// Keys of a CTA: [lo, hi) of the request's cached rows (places in its ring, or positions); lo is a multiple of 16
struct Range {
    int slot, pos, lo, hi, seen;         // seen: first visible row
    int current;                         // row of the new token, which the kernel before these two stores
    __device__ __forceinline__ Range(const pa::Step& a, int b, int split, int splits) {
        slot = a.slots[b], pos = a.pos[b];
        const bool ring = a.c.table == nullptr;
        const int nk = ring ? min(pos + 1, a.c.cap) : pos + 1;
        seen = !ring && a.window > 0 ? max(0, nk - a.window) : 0;
        current = ring ? pos % a.c.cap : pos;
        const int first = seen / 16 * 16, per = ((nk - first + splits - 1) / splits + STEP - 1) / STEP * STEP;
        lo = first + split * per, hi = min(nk, lo + per);
    }
    // row of the cache buffers; 16 rows from a multiple of 16 lie in one page, and in a ring they follow one another
    __device__ __forceinline__ long long row(const pa::Cache& c, int key) const {
        return c.table == nullptr ? (long long)slot * c.cap + key : (long long)c.table[(long long)slot * c.table_ld + key / pa::PAGE] * pa::PAGE + key % pa::PAGE;
    }
    // may the 16 keys from key0 be read while the kernel that stores the new token runs?
    __device__ __forceinline__ bool early(int key0) const { return key0 < hi && (current < key0 || current >= key0 + 16); }
};

// grid (splits, G * head tiles, n).  KG: groups of 32 key dims
template <int KG>
__global__ void __launch_bounds__(WARPS * 32) talk_scores_kernel(Args t) {
    const pa::Step& a = t.s;
    __shared__ float ml[WARPS][HEADS][2];
    const int w = threadIdx.x >> 5, l = threadIdx.x & 31, g = l >> 2, q = l & 3;
    const int splits = gridDim.x, split = blockIdx.x, b = blockIdx.z;
    const int qpg = a.H / a.G, tiles = (qpg + HEADS - 1) / HEADS;
    const int hk = blockIdx.y / tiles, h0 = hk * qpg + (blockIdx.y % tiles) * HEADS;
    const int nh = min(HEADS, hk * qpg + qpg - h0);
    const Range r(a, b, split, splits);
    const uint4 zero = make_uint4(0, 0, 0, 0);
    auto load_k = [&](uint4 (&kf)[2][KG], int key0) {
        const bf16* p = (const bf16*)a.c.k + (r.row(a.c, key0) * a.G + hk) * a.dk;
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int i = g + 8 * e;
#pragma unroll
            for (int c = 0; c < KG; ++c) {
                const int d = c * 32 + q * 8;
                kf[e][c] = key0 + i < r.hi && d < a.dk ? __ldcs(reinterpret_cast<const uint4*>(p + (long long)i * a.G * a.dk + d)) : zero;
            }
        }
    };
    uint4 kf[2][KG];
    int key0 = r.lo + 16 * w;
    const bool early = r.early(key0);
    if (early) load_k(kf, key0);
    asm volatile("griddepcontrol.wait;" ::: "memory");
    pdl_trigger();                                           // behind the wait: the kernel behind this one reads the cache early, too
    if (!early && key0 < r.hi) load_k(kf, key0);
    uint4 qf[KG];                                            // head h0 + g
#pragma unroll
    for (int c = 0; c < KG; ++c) {
        const int d = c * 32 + q * 8;
        qf[c] = g < nh && d < a.dk ? *reinterpret_cast<const uint4*>((const bf16*)a.q + (long long)b * a.ldq + (h0 + g) * a.dk + d) : zero;
    }
    const float sc = a.scale * LOG2E;
    float* out = t.scores + ((long long)b * a.H + h0) * t.lds;
    float m[2] = {-INFINITY, -INFINITY}, sum[2] = {0.f, 0.f};            // heads 2q, 2q + 1 over this lane's keys
    for (; key0 < r.hi; key0 += STEP) {
        float s[4] = {0.f, 0.f, 0.f, 0.f};                   // (key g, key g + 8) x (head 2q, head 2q + 1)
#pragma unroll
        for (int c = 0; c < KG; ++c) {
            const uint32_t f1[4] = {kf[0][c].x, kf[1][c].x, kf[0][c].y, kf[1][c].y};
            const uint32_t f2[4] = {kf[0][c].z, kf[1][c].z, kf[0][c].w, kf[1][c].w};
            mma16816(s, f1, qf[c].x, qf[c].y);
            mma16816(s, f2, qf[c].z, qf[c].w);
        }
        if (key0 + STEP < r.hi) load_k(kf, key0 + STEP);
#pragma unroll
        for (int e = 0; e < 2; ++e) {                        // head
            float x[2];
#pragma unroll
            for (int k = 0; k < 2; ++k) {                    // key
                const int key = key0 + g + 8 * k;
                x[k] = key >= r.seen && key < r.hi ? s[2 * k + e] * sc : -INFINITY;
                if (key < r.hi && 2 * q + e < nh) out[(2 * q + e) * t.lds + key] = x[k];
            }
            const float mx = fmaxf(m[e], fmaxf(x[0], x[1]));
            if (mx != -INFINITY) sum[e] = sum[e] * ex2(m[e] - mx) + ex2(x[0] - mx) + ex2(x[1] - mx);
            m[e] = mx;
        }
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
#pragma unroll
        for (int x = 4; x < 32; x <<= 1) {                   // over the lanes with the same q
            const float mo = __shfl_xor_sync(0xffffffffu, m[e], x), so = __shfl_xor_sync(0xffffffffu, sum[e], x), mx = fmaxf(m[e], mo);
            if (mx != -INFINITY) sum[e] = sum[e] * ex2(m[e] - mx) + so * ex2(mo - mx);
            m[e] = mx;
        }
        if (g == 0) {
            ml[w][2 * q + e][0] = m[e];
            ml[w][2 * q + e][1] = sum[e];
        }
    }
    __syncthreads();
    if (threadIdx.x < nh) {
        float mx = -INFINITY, s = 0.f;
#pragma unroll
        for (int k = 0; k < WARPS; ++k) mx = fmaxf(mx, ml[k][threadIdx.x][0]);
        if (mx != -INFINITY) {
#pragma unroll
            for (int k = 0; k < WARPS; ++k) s += ml[k][threadIdx.x][1] * ex2(ml[k][threadIdx.x][0] - mx);
        }
        *reinterpret_cast<float2*>(t.parts + (((long long)b * a.H + h0 + threadIdx.x) * splits + split) * 2) = make_float2(mx, s);
    }
}

// grid (splits, G * head tiles, n), cluster (splits, 1, 1).  VG: groups of 64 value dims
template <int VG>
__global__ void __launch_bounds__(WARPS * 32) talk_values_kernel(Args t) {
    const pa::Step& a = t.s;
    constexpr int DV = VG * 64;
    extern __shared__ float dyn[];
    __shared__ float part[WARPS][HEADS][DV];
    __shared__ float sum[HEADS][DV];
    const int HP = (a.H + 7) / 8 * 8;                        // softmax heads, padded with coefficients of zero
    float* coef = dyn;                                       // [HP][HEADS]: T[h0 + n, g] / sum of g
    float* top = dyn + HP * HEADS;                           // [HP] maximum of head g
    const int w = threadIdx.x >> 5, l = threadIdx.x & 31, g = l >> 2, q = l & 3;
    const int splits = gridDim.x, split = blockIdx.x, b = blockIdx.z;
    const int qpg = a.H / a.G, tiles = (qpg + HEADS - 1) / HEADS;
    const int hk = blockIdx.y / tiles, h0 = hk * qpg + (blockIdx.y % tiles) * HEADS;
    const int nh = min(HEADS, hk * qpg + qpg - h0);
    const Range r(a, b, split, splits);
    const uint4 zero = make_uint4(0, 0, 0, 0);
    auto load_v = [&](uint4 (&vf)[4][VG], int key0) {
        const bf16* p = (const bf16*)a.c.v + (r.row(a.c, key0) * a.G + hk) * a.dv;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = 2 * q + (e & 1) + 8 * (e >> 1);
#pragma unroll
            for (int c = 0; c < VG; ++c) {
                const int d = c * 64 + g * 8;
                vf[e][c] = key0 + i < r.hi && d < a.dv ? __ldcs(reinterpret_cast<const uint4*>(p + (long long)i * a.G * a.dv + d)) : zero;
            }
        }
    };
    uint4 vf[4][VG];
    int key0 = r.lo + 16 * w;
    const bool early = r.early(key0);
    if (early) load_v(vf, key0);
    pdl_trigger();
    asm volatile("griddepcontrol.wait;" ::: "memory");
    if (!early && key0 < r.hi) load_v(vf, key0);
    for (int i = threadIdx.x; i < HP; i += WARPS * 32) {
        float mx = -INFINITY, s = 0.f;
        if (i < a.H) {
            const float2* p = reinterpret_cast<const float2*>(t.parts) + ((long long)b * a.H + i) * splits;
            for (int k = 0; k < splits; ++k) mx = fmaxf(mx, p[k].x);
            for (int k = 0; k < splits; ++k) s += p[k].x == -INFINITY ? 0.f : p[k].y * ex2(p[k].x - mx);
        }
        top[i] = i < a.H ? mx : 0.f;
        const float inv = i < a.H ? 1.f / s : 0.f;
#pragma unroll
        for (int n = 0; n < HEADS; ++n) coef[i * HEADS + n] = i < a.H && n < nh ? t.table[(long long)(h0 + n) * a.H + i] * inv : 0.f;
    }
    __syncthreads();
    const float* sc = t.scores + (long long)b * a.H * t.lds;
    float o[VG * 4][4];
#pragma unroll
    for (int i = 0; i < VG * 4; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    for (; key0 < r.hi; key0 += STEP) {
        float p[4] = {0.f, 0.f, 0.f, 0.f};                   // mixed weights: (key g, key g + 8) x (head 2q, head 2q + 1)
        const bool in0 = key0 + g < r.hi, in1 = key0 + g + 8 < r.hi;
#pragma unroll 2
        for (int c = 0; c < HP; c += 8) {
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {                    // (key g + 8 (e & 1), softmax head c + q + 4 (e >> 1))
                const int head = c + q + 4 * (e >> 1);
                float x = 0.f;
                if ((e & 1 ? in1 : in0) && head < a.H) x = ex2(sc[head * t.lds + key0 + g + 8 * (e & 1)] - top[head]);
                hi[e] = tf32(x);
                lo[e] = tf32(x - __uint_as_float(hi[e]));
            }
            const float c0 = coef[(c + q) * HEADS + g], c1 = coef[(c + q + 4) * HEADS + g];
            const uint32_t b0 = tf32(c0), b1 = tf32(c1);
            const uint32_t d0 = tf32(c0 - __uint_as_float(b0)), d1 = tf32(c1 - __uint_as_float(b1));
            mma1688(p, lo, b0, b1);
            mma1688(p, hi, d0, d1);
            mma1688(p, hi, b0, b1);
        }
        const uint32_t b0 = transpose8x8(pack2(p[0], p[1])), b1 = transpose8x8(pack2(p[2], p[3]));
#pragma unroll
        for (int i = 0; i < VG; ++i)
#pragma unroll
            for (int x = 0; x < 4; ++x) {                    // rows g, g + 8 of the tile: dims 2x, 2x + 1 of this lane's eight
                const uint32_t w0 = word(vf[0][i], x), w1 = word(vf[1][i], x), w2 = word(vf[2][i], x), w3 = word(vf[3][i], x);
                const uint32_t f[4] = {__byte_perm(w0, w1, 0x5410), __byte_perm(w0, w1, 0x7632), __byte_perm(w2, w3, 0x5410),
                                       __byte_perm(w2, w3, 0x7632)};
                mma16816(o[i * 4 + x], f, b0, b1);
            }
        if (key0 + STEP < r.hi) load_v(vf, key0 + STEP);
    }
#pragma unroll
    for (int i = 0; i < VG; ++i)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const int d = i * 64 + g * 8 + 2 * x;
            part[w][2 * q][d] = o[i * 4 + x][0];
            part[w][2 * q + 1][d] = o[i * 4 + x][1];
            part[w][2 * q][d + 1] = o[i * 4 + x][2];
            part[w][2 * q + 1][d + 1] = o[i * 4 + x][3];
        }
    __syncthreads();
    for (int i = threadIdx.x; i < HEADS * DV; i += WARPS * 32) {
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
        float y = 0.f;
        for (int k = 0; k < splits; ++k) y += cluster.map_shared_rank(&sum[0][0], k)[h * DV + d];
        ((bf16*)a.out)[(long long)b * a.ldo + (long long)(h0 + h) * a.dv + d] = __float2bfloat16(y);
    }
    cluster.sync();                                          // nobody leaves while its shared memory is read
}

template <typename Kernel>
static int launch_one(Kernel kernel, const Args& t, int splits, bool cluster, size_t smem, cudaStream_t st) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(splits, t.s.G * ((t.s.H / t.s.G + HEADS - 1) / HEADS), t.s.n);
    cfg.blockDim = dim3(WARPS * 32);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = splits;
    attr[1].val.clusterDim.y = 1;
    attr[1].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = cluster ? 2 : 1;
    return (int)cudaLaunchKernelEx(&cfg, kernel, t);
}

template <int KG, int VG>
static int launch(const Args& t, int splits, cudaStream_t st) {
    const int rc = launch_one(talk_scores_kernel<KG>, t, splits, false, 0, st);
    return rc ? rc : launch_one(talk_values_kernel<VG>, t, splits, true, sizeof(float) * ((t.s.H + 7) / 8 * 8) * (HEADS + 1), st);
}

}  // namespace ts
}  // namespace lmoe

using namespace lmoe;

// bf16, head sizes multiples of 16 up to 128, up to 256 heads, 16-byte aligned bases, pitches multiples of 8; scores has room for every
// cached row of a request (lds); splits: 1, 2, 4 or 8 CTAs per (request, heads).  Slots, positions and the page table must have been on
// the device before the kernel that precedes these in the stream was launched; that kernel stores the new token.
LMOE_API int lmoe_talk_step(const ts::Args* tp, int splits, cudaStream_t st) {
    const ts::Args& t = *tp;
    const pa::Step& a = t.s;
    if (a.n <= 0 || a.G <= 0 || a.H <= 0 || a.H > 256 || a.H % a.G || a.dk <= 0 || a.dv <= 0 || a.dk % 16 || a.dv % 16 || a.dk > 128 || a.dv > 128 || a.ldq % 8 ||
        !(a.scale > 0.f) || (a.c.table == nullptr && a.c.cap <= 0) || t.lds <= 0 || t.table == nullptr || t.scores == nullptr || t.parts == nullptr ||
        ((reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(a.c.k) | reinterpret_cast<uintptr_t>(a.c.v)) & 15) ||
        (splits != 1 && splits != 2 && splits != 4 && splits != 8))
        return -1;
    if (a.dk <= 64) return a.dv <= 64 ? ts::launch<2, 1>(t, splits, st) : ts::launch<2, 2>(t, splits, st);
    return a.dv <= 64 ? ts::launch<4, 1>(t, splits, st) : ts::launch<4, 2>(t, splits, st);
}
