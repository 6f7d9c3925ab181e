// One-token softmax attention over cached keys for bf16: grouped-query layers with a ring or pages, and latent layers, whose
// cached row is key and value at once (then it is read once).  Arguments and cache addressing: packed_attn.cuh.  The new token's key
// and value are in the cache already; the order of the keys does not matter to a softmax, so a ring needs no unrolling.
//
// A CTA takes 16 or 32 query heads of one kv head and a range of keys; the CTAs of a cluster share the keys of a request.
//   cp.async   tiles of 64 keys (one page), two stages
//   scores     a warp owns 8 keys of the tile: mma.sync, queries as the A operand, keys straight from the row-major tile
//   softmax    online, 256 threads over [heads x 64], probabilities to shared memory in bf16
//   values     a warp owns 16-column strips of the output, fragments of V by transposing ldmatrix, accumulators in registers
// The partial results of a cluster meet in distributed shared memory.
#include <cooperative_groups.h>

#include "attn_math.cuh"
#include "mma_utils.cuh"
#include "packed_attn.cuh"

namespace lmoe {
namespace pas {
namespace cg = cooperative_groups;
using pa::Step;

constexpr int THREADS = 256, WARPS = 8, KT = pa::PAGE;
constexpr float LOG2E = 1.4426950408889634f;

struct Layout {                          // offsets in bytes inside the dynamic shared memory
    int k_ld, v_ld, q, k, v, stage, s, p, ml, total;
    // row lengths of an odd number of 16-byte pieces: ldmatrix rows fall into different banks
    __host__ __device__ static int pad(int d) { return d + ((d / 8) % 2 == 0 ? 8 : 0); }
    __host__ __device__ Layout(int mt, int dk, int dv, bool shared) {
        const int rows = 16 * mt;
        k_ld = pad(dk);
        v_ld = shared ? k_ld : pad(dv);
        q = 0;
        k = q + rows * k_ld * 2;
        v = shared ? 0 : KT * k_ld * 2;                      // inside a stage
        stage = KT * (k_ld + (shared ? 0 : v_ld)) * 2;
        const int out = rows * (dv + 4) * 4;                 // the result takes the place of the stages
        s = k + (2 * stage > out ? 2 * stage : out) + 64;    // ldmatrix of the last 16 columns may read past a row's end
        p = s + rows * (KT + 4) * 4;
        ml = p + rows * (KT + 8) * 2;
        total = ml + 3 * rows * 4;
    }
};

// MT: tiles of 16 heads, NP: 16-column strips of the output per warp
template <int MT, int NP, bool SHARED>
__global__ void __launch_bounds__(THREADS) packed_attn_step_kernel(Step a) {
    extern __shared__ __align__(128) unsigned char smem[];
    constexpr int ROWS = 16 * MT, TPR = THREADS / ROWS, KPT = KT / TPR;     // threads per row, keys per thread in the softmax
    const Layout L(MT, a.dk, a.dv, SHARED);
    bf16* Q = reinterpret_cast<bf16*>(smem + L.q);
    float* S = reinterpret_cast<float*>(smem + L.s);
    bf16* P = reinterpret_cast<bf16*>(smem + L.p);
    float* ML = reinterpret_cast<float*>(smem + L.ml);       // [ROWS] maximum (log2 units), sum, correction of the current tile
    const int w = threadIdx.x >> 5, l = threadIdx.x & 31, g = l >> 2, q = l & 3;
    const int splits = gridDim.x, split = blockIdx.x, b = blockIdx.z;
    const int qpg = a.H / a.G, tiles_h = (qpg + ROWS - 1) / ROWS;
    const int hk = blockIdx.y / tiles_h, h0 = hk * qpg + (blockIdx.y % tiles_h) * ROWS;
    const int nh = min(ROWS, hk * qpg + qpg - h0);
    // slots and positions are older than the kernel before this one
    const int slot = a.slots[b], pos = a.pos[b];
    const bool ring = a.c.table == nullptr;
    const int nk = ring ? min(pos + 1, a.c.cap) : pos + 1;   // cached rows to read: [lo, nk)
    const int lo = !ring && a.window > 0 ? max(0, nk - a.window) : 0;
    const int t_lo = lo / KT, n_t = (nk + KT - 1) / KT - t_lo, per = (n_t + splits - 1) / splits;
    const int t_beg = t_lo + split * per, t_end = min(t_lo + n_t, t_beg + per);

    auto load = [&](int t) {
        const int stage = (t - t_beg) & 1, r0 = t * KT;
        const long long row = ring ? (long long)slot * a.c.cap + r0 : (long long)a.c.table[(long long)slot * a.c.table_ld + t] * KT;
        bf16* Ks = reinterpret_cast<bf16*>(smem + L.k + stage * L.stage);
        const bf16* kc = (const bf16*)a.c.k + (row * a.G + hk) * a.dk;
        const int kp = a.dk / 8;
        for (int i = threadIdx.x; i < KT * kp; i += THREADS) {
            const int j = i / kp, c = (i % kp) * 8;
            const bool ok = r0 + j < nk;
            cp_async16(Ks + j * L.k_ld + c, ok ? kc + (long long)j * a.G * a.dk + c : kc, ok);
        }
        if (!SHARED) {
            bf16* Vs = reinterpret_cast<bf16*>(smem + L.k + stage * L.stage + L.v);
            const bf16* vc = (const bf16*)a.c.v + (row * a.G + hk) * a.dv;
            const int vp = a.dv / 8;
            for (int i = threadIdx.x; i < KT * vp; i += THREADS) {
                const int j = i / vp, c = (i % vp) * 8;
                const bool ok = r0 + j < nk;
                cp_async16(Vs + j * L.v_ld + c, ok ? vc + (long long)j * a.G * a.dv + c : vc, ok);
            }
        }
    };

    // While the kernel before this one (it stores the new token's key) still runs: tiles that do not hold that token
    const int t_cur = (ring ? pos % a.c.cap : pos) / KT;
    const bool early0 = t_beg < t_end && t_beg != t_cur, early1 = t_beg + 1 < t_end && t_beg + 1 != t_cur && early0;
    if (early0) load(t_beg);
    cp_async_commit();
    if (early1) load(t_beg + 1);
    if (early1) cp_async_commit();
    pdl_trigger();
    asm volatile("griddepcontrol.wait;" ::: "memory");
    // a first tile that had to wait joins the second group; waiting for all groups below covers it
    if (t_beg < t_end && !early0) load(t_beg);
    if (t_beg + 1 < t_end && !early1) load(t_beg + 1);
    if (!early1) cp_async_commit();
    bool first_late = !early0;
    {
        const bf16* qg = (const bf16*)a.q + (long long)b * a.ldq + (long long)h0 * a.dk;
        const int kp = a.dk / 8;
        for (int i = threadIdx.x; i < ROWS * kp; i += THREADS) {
            const int h = i / kp, c = (i % kp) * 8;
            *reinterpret_cast<uint4*>(Q + h * L.k_ld + c) = h < nh ? *reinterpret_cast<const uint4*>(qg + h * a.dk + c) : make_uint4(0, 0, 0, 0);
        }
    }
    const float sc = a.scale * LOG2E;
    const int srow = threadIdx.x / TPR, sk0 = (threadIdx.x % TPR) * KPT;    // this thread's row and first key in the softmax
    float m = -INFINITY, sum = 0.f;
    float o[MT][2 * NP][4];
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int j = 0; j < 2 * NP; ++j) o[i][j][0] = o[i][j][1] = o[i][j][2] = o[i][j][3] = 0.f;

    for (int t = t_beg; t < t_end; ++t) {
        if (first_late) cp_async_wait<0>();                   // (once) both tiles are in the same group
        else cp_async_wait<1>();
        first_late = false;
        __syncthreads();
        const bf16* Ks = reinterpret_cast<const bf16*>(smem + L.k + ((t - t_beg) & 1) * L.stage);
        const bf16* Vs = SHARED ? Ks : reinterpret_cast<const bf16*>(smem + L.k + ((t - t_beg) & 1) * L.stage + L.v);
        {
            float s[MT][2][4];
#pragma unroll
            for (int i = 0; i < MT; ++i)
#pragma unroll
                for (int e = 0; e < 2; ++e) s[i][e][0] = s[i][e][1] = s[i][e][2] = s[i][e][3] = 0.f;
            const bf16* kr = Ks + (8 * w + (l & 7)) * L.k_ld + 8 * (l >> 3);
#pragma unroll 2
            for (int k0 = 0; k0 < a.dk; k0 += 32) {
                uint32_t kb[4], qa[4];
                ldsm_x4(kb, kr + k0);
#pragma unroll
                for (int i = 0; i < MT; ++i) {
                    load_a(qa, Q, L.k_ld, 16 * i, k0);
                    mma16816(s[i][0], qa, kb[0], kb[1]);
                }
                if (k0 + 16 < a.dk) {
#pragma unroll
                    for (int i = 0; i < MT; ++i) {
                        load_a(qa, Q, L.k_ld, 16 * i, k0 + 16);
                        mma16816(s[i][1], qa, kb[2], kb[3]);
                    }
                }
            }
#pragma unroll
            for (int i = 0; i < MT; ++i) {
                float* sr = S + (16 * i + g) * (KT + 4) + 8 * w + 2 * q;
                *reinterpret_cast<float2*>(sr) = make_float2(s[i][0][0] + s[i][1][0], s[i][0][1] + s[i][1][1]);
                *reinterpret_cast<float2*>(sr + 8 * (KT + 4)) = make_float2(s[i][0][2] + s[i][1][2], s[i][0][3] + s[i][1][3]);
            }
        }
        __syncthreads();
        {
            const float* sr = S + srow * (KT + 4) + sk0;
            float x[KPT], mx = m;
#pragma unroll
            for (int i = 0; i < KPT; i += 4) {
                const float4 f = *reinterpret_cast<const float4*>(sr + i);
                x[i] = f.x; x[i + 1] = f.y; x[i + 2] = f.z; x[i + 3] = f.w;
            }
#pragma unroll
            for (int i = 0; i < KPT; ++i) {
                const int key = t * KT + sk0 + i;
                x[i] = key >= lo && key < nk ? x[i] * sc : -INFINITY;
                mx = fmaxf(mx, x[i]);
            }
#pragma unroll
            for (int d = 1; d < TPR; d <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
            const float corr = m == -INFINITY ? 0.f : ex2(m - mx);       // a tile of [lo, nk) has a visible key: mx is finite
            float ps = 0.f;
#pragma unroll
            for (int i = 0; i < KPT; ++i) {
                x[i] = ex2(x[i] - mx);
                ps += x[i];
            }
#pragma unroll
            for (int i = 0; i < KPT; i += 2)
                *reinterpret_cast<__nv_bfloat162*>(P + srow * (KT + 8) + sk0 + i) = __floats2bfloat162_rn(x[i], x[i + 1]);
#pragma unroll
            for (int d = 1; d < TPR; d <<= 1) ps += __shfl_xor_sync(0xffffffffu, ps, d);
            sum = sum * corr + ps;
            m = mx;
            if (sk0 == 0) ML[2 * ROWS + srow] = corr;
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < MT; ++i) {
            const float c0 = ML[2 * ROWS + 16 * i + g], c1 = ML[2 * ROWS + 16 * i + g + 8];
#pragma unroll
            for (int j = 0; j < 2 * NP; ++j) {
                o[i][j][0] *= c0; o[i][j][1] *= c0;
                o[i][j][2] *= c1; o[i][j][3] *= c1;
            }
        }
#pragma unroll
        for (int k0 = 0; k0 < KT; k0 += 16) {
            uint32_t pf[MT][4];
#pragma unroll
            for (int i = 0; i < MT; ++i) load_a(pf[i], P, KT + 8, 16 * i, k0);
#pragma unroll
            for (int j = 0; j < NP; ++j) {
                const int n0 = (w + WARPS * j) * 16;
                if (n0 < a.dv) {
                    uint32_t vb[4];
                    load_b2_t(vb, Vs, L.v_ld, n0, k0);
#pragma unroll
                    for (int i = 0; i < MT; ++i) {
                        mma16816(o[i][2 * j], pf[i], vb[0], vb[1]);
                        mma16816(o[i][2 * j + 1], pf[i], vb[2], vb[3]);
                    }
                }
            }
        }
        __syncthreads();
        if (t + 2 < t_end) load(t + 2);
        cp_async_commit();
    }
    cp_async_wait<0>();
    __syncthreads();
    // join the cluster: every CTA finishes a slice of the (head, column) pairs
    float* O = reinterpret_cast<float*>(smem + L.k);         // [ROWS][dv + 4]
    const int o_ld = a.dv + 4;
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int j = 0; j < NP; ++j) {
            const int n0 = (w + WARPS * j) * 16;
            if (n0 < a.dv) {
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    float* p = O + (16 * i + g) * o_ld + n0 + 8 * e + 2 * q;
                    *reinterpret_cast<float2*>(p) = make_float2(o[i][2 * j + e][0], o[i][2 * j + e][1]);
                    *reinterpret_cast<float2*>(p + 8 * o_ld) = make_float2(o[i][2 * j + e][2], o[i][2 * j + e][3]);
                }
            }
        }
    if (sk0 == 0) {
        ML[srow] = m;
        ML[ROWS + srow] = sum;
    }
    auto cluster = cg::this_cluster();
    cluster.sync();
    const int vp = a.dv / 4;
    for (int i = split * THREADS + threadIdx.x; i < nh * vp; i += splits * THREADS) {
        const int h = i / vp, d = (i % vp) * 4;
        float mx = -INFINITY;
        for (int r = 0; r < splits; ++r) mx = fmaxf(mx, cluster.map_shared_rank(ML, r)[h]);
        float ls = 0.f;
        float4 os = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int r = 0; r < splits; ++r) {
            const float* ml = cluster.map_shared_rank(ML, r);
            const float f = ml[h] == -INFINITY ? 0.f : ex2(ml[h] - mx);
            const float4 x = *reinterpret_cast<const float4*>(cluster.map_shared_rank(O, r) + h * o_ld + d);
            ls += ml[ROWS + h] * f;
            os.x += x.x * f; os.y += x.y * f; os.z += x.z * f; os.w += x.w * f;
        }
        const float inv = 1.f / ls;
        __nv_bfloat162 y[2] = {__floats2bfloat162_rn(os.x * inv, os.y * inv), __floats2bfloat162_rn(os.z * inv, os.w * inv)};
        *reinterpret_cast<uint2*>((bf16*)a.out + (long long)b * a.ldo + (long long)(h0 + h) * a.dv + d) = *reinterpret_cast<uint2*>(y);
    }
    cluster.sync();                                          // nobody leaves while its shared memory is read
}

template <int MT, int NP, bool SHARED>
static int launch(const Step& a, int splits, cudaStream_t st) {
    const int smem = Layout(MT, a.dk, a.dv, SHARED).total;
    if (smem > 227 * 1024) return -2;
    auto kern = packed_attn_step_kernel<MT, NP, SHARED>;
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e == cudaSuccess && splits > 8) e = cudaFuncSetAttribute(kern, cudaFuncAttributeNonPortableClusterSizeAllowed, 1);
    if (e != cudaSuccess) return (int)e;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(splits, a.G * ((a.H / a.G + 16 * MT - 1) / (16 * MT)), a.n);
    cfg.blockDim = dim3(THREADS);
    cfg.dynamicSmemBytes = smem;
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
    return (int)cudaLaunchKernelEx(&cfg, kern, a);
}

template <int NP, bool SHARED>
static int by_heads(const Step& a, int splits, cudaStream_t st) {
    return a.H / a.G > 16 ? launch<2, NP, SHARED>(a, splits, st) : launch<1, NP, SHARED>(a, splits, st);
}

template <bool SHARED>
static int by_width(const Step& a, int splits, cudaStream_t st) {
    if (a.dv <= 128) return by_heads<1, SHARED>(a, splits, st);
    if (a.dv <= 256) return by_heads<2, SHARED>(a, splits, st);
    return by_heads<4, SHARED>(a, splits, st);
}

}  // namespace pas
}  // namespace lmoe

using namespace lmoe;

// bf16, head sizes multiples of 16, values up to 512 wide, 16-byte aligned bases, pitches multiples of 8; a.c.v == a.c.k (and dv ==
// dk): the rows are key and value at once.  splits: 1, 2, 4, 8 or 16 CTAs per (request, heads).  Slots, positions and the page table
// must have been on the device before the kernel that precedes this one in the stream was launched; that kernel stores the new token.
// Returns -2 when the head sizes do not fit shared memory.
LMOE_API int lmoe_packed_attn_step(const pa::Step* ap, int splits, cudaStream_t st) {
    const pa::Step& a = *ap;
    if (a.n <= 0 || a.G <= 0 || a.H <= 0 || a.H % a.G || a.dk <= 0 || a.dv <= 0 || a.dk % 16 || a.dv % 16 || a.dv > 512 || a.ldq % 8 || a.ldo % 8 ||
        !(a.scale > 0.f) || (a.c.table == nullptr && a.c.cap <= 0) ||
        ((reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(a.c.k) | reinterpret_cast<uintptr_t>(a.c.v) |
          reinterpret_cast<uintptr_t>(a.out)) & 15) ||
        (splits != 1 && splits != 2 && splits != 4 && splits != 8 && splits != 16))
        return -1;
    if (a.c.v == a.c.k) return a.dk != a.dv ? -1 : pas::by_width<true>(a, splits, st);
    return pas::by_width<false>(a, splits, st);
}
