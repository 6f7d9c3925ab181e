// One-token attention (softmax, or sigmoid weights of every key by itself) over cached keys for bf16: grouped-query layers with a ring or pages, and latent layers, whose
// cached row is key and value at once (then it is read once).  Arguments and cache addressing: packed_attn.cuh.  The new token's key
// and value are in the cache already; the order of the keys does not matter to a softmax, so a ring needs no unrolling.
//
// A CTA takes 16 query heads of one kv head and a range of keys; the CTAs of a cluster share the keys of a request.  Two CTAs per SM
// hide each other's barriers.
//   loads      tiles of 64 keys (32 where rows are wide) by TMA (128-byte swizzle), 2 - 4 stages counted by mbarriers
//   scores     a warp owns every eighth step of 16 along the head dimension: mma.sync, queries as the A operand
//   softmax    online, 256 threads over [16 heads x keys] add the warps' partial scores; probabilities to shared memory in bf16
//   values     a warp owns 16-column strips of the output, fragments of V by transposing ldmatrix, accumulators in registers
// The values of a tile and the scores of the next one run between the same two barriers.  The partial results of a cluster meet in
// distributed shared memory.  Waits are bounded (status word `err`).
#include <cooperative_groups.h>

#include "attn_math.cuh"
#include "flash_tc_utils.cuh"
#include "mma_utils.cuh"
#include "packed_attn.cuh"

namespace lmoe {
namespace pas {
namespace cg = cooperative_groups;
using pa::Step;

constexpr int THREADS = 256, WARPS = 8, ROWS = 16, MAX_STAGES = 4, MAX_SPLITS = 16;
constexpr int TPR = THREADS / ROWS;                          // threads per row in the softmax
constexpr float LOG2E = 1.4426950408889634f;

struct Layout {                          // offsets in bytes inside the dynamic shared memory (after alignment to 1024)
    int q_ld, v, stage, q, s, p, ml, total;
    __host__ __device__ Layout(int KT, int dk, int dv, bool shared, int stages) {
        const int kb = (dk + 63) / 64, vb = (dv + 63) / 64;
        q_ld = dk + ((dk / 8) % 2 == 0 ? 8 : 0);             // an odd number of 16-byte pieces: ldmatrix rows fall into different banks
        v = shared ? 0 : kb * KT * 128;                      // inside a stage
        stage = (kb + (shared ? 0 : vb)) * KT * 128;
        const int out = ROWS * (dv + 4) * 4;                 // the result takes the place of the stages
        q = stages * stage > out ? stages * stage : (out + 15) / 16 * 16;
        s = q + ROWS * q_ld * 2;
        p = s + WARPS * ROWS * (KT + 4) * 4;
        ml = p + ROWS * (KT + 8) * 2;
        total = ml + 3 * ROWS * 4 + 1024;
    }
};

// KT: keys per tile; N: 128-column groups of keys and values (a warp has one step of 16 of each)
template <int KT, int N, bool SHARED>
__global__ void __launch_bounds__(THREADS, 2)
packed_attn_step_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV, Step a, int stages, int* err) {
    constexpr int KE = KT / 16, KPT = KT / TPR;              // 16-key groups, keys per thread in the softmax
    static_assert(pa::PAGE % KT == 0 && KPT % 2 == 0, "tiles inside a page");
    extern __shared__ unsigned char smem_raw[];
    unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    __shared__ uint64_t full[MAX_STAGES];
    __shared__ float part[2][MAX_SPLITS][ROWS];              // maxima and sums of the cluster's CTAs
    __shared__ int abort_flag;
    const Layout L(KT, a.dk, a.dv, SHARED, stages);
    bf16* Q = reinterpret_cast<bf16*>(smem + L.q);
    float* S = reinterpret_cast<float*>(smem + L.s);
    bf16* P = reinterpret_cast<bf16*>(smem + L.p);
    float* ML = reinterpret_cast<float*>(smem + L.ml);       // [ROWS] maximum (log2 units), sum, correction of the current tile
    const int w = threadIdx.x >> 5, l = threadIdx.x & 31, g = l >> 2, q = l & 3;
    const int splits = gridDim.x, split = blockIdx.x, b = blockIdx.z;
    const int qpg = a.H / a.G, tiles_h = (qpg + ROWS - 1) / ROWS;
    const int hk = blockIdx.y / tiles_h, h0 = hk * qpg + (blockIdx.y % tiles_h) * ROWS;
    const int nh = min(ROWS, hk * qpg + qpg - h0);
    // slots, positions and page numbers are older than the kernel before this one
    const int slot = a.slots[b], pos = a.pos[b];
    const bool ring = a.c.table == nullptr;
    const int nk = ring ? min(pos + 1, a.c.cap) : pos + 1;   // cached rows to read: [lo, nk)
    const int lo = !ring && a.window > 0 ? max(0, nk - a.window) : 0;
    const int t_lo = lo / KT, n_t = (nk + KT - 1) / KT - t_lo, per = (n_t + splits - 1) / splits;
    const int t_beg = t_lo + split * per, t_end = min(t_lo + n_t, t_beg + per);

    if (threadIdx.x == 0) {
        for (int i = 0; i < MAX_STAGES; ++i) tc::mbar_init(&full[i], 1);
        abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    auto load = [&](int t, int st) {                         // one thread
        const int row = ring ? slot * a.c.cap + t * KT
                             : a.c.table[(long long)slot * a.c.table_ld + t / (pa::PAGE / KT)] * pa::PAGE + t % (pa::PAGE / KT) * KT;
        unsigned char* dst = smem + st * L.stage;
        tc::mbar_expect_tx(&full[st], (uint32_t)L.stage);
        for (int c = 0; c * 64 < a.dk; ++c) fatc::tma_load_4d(dst + c * KT * 128, &tmK, &full[st], c * 64, hk, row, 0);
        if (!SHARED)
            for (int c = 0; c * 64 < a.dv; ++c) fatc::tma_load_4d(dst + L.v + c * KT * 128, &tmV, &full[st], c * 64, hk, row, 0);
    };

    // While the kernel before this one (it stores the new token's key) still runs: the tiles in front of the one with that token
    const int t_cur = (ring ? pos % a.c.cap : pos) / KT, ahead = min(t_end, t_beg + stages);
    int t_in = t_beg;
    if (threadIdx.x == 0)
        for (; t_in < ahead && t_in != t_cur; ++t_in) load(t_in, t_in - t_beg);
    pdl_trigger();
    asm volatile("griddepcontrol.wait;" ::: "memory");
    if (threadIdx.x == 0)
        for (; t_in < ahead; ++t_in) load(t_in, t_in - t_beg);
    {
        const bf16* qg = (const bf16*)a.q + (long long)b * a.ldq + (long long)h0 * a.dk;
        for (int h = w; h < ROWS; h += WARPS)
            for (int c = l * 8; c < a.dk; c += 256)
                *reinterpret_cast<uint4*>(Q + h * L.q_ld + c) = h < nh ? *reinterpret_cast<const uint4*>(qg + h * a.dk + c) : make_uint4(0, 0, 0, 0);
    }
    __syncthreads();
    const float sc = a.scale * LOG2E;
    const int bufs = min(WARPS, a.dk / 16);                  // warps with a step of the head dimension
    const int srow = threadIdx.x / TPR, sk0 = (threadIdx.x % TPR) * KPT;    // this thread's row and first key in the softmax
    const bool sigmoid = a.bias != nullptr;                  // then there is no maximum to follow: m stays 0
    const float head_bias = sigmoid && srow < nh ? a.bias[h0 + srow] * LOG2E : 0.f;
    float m = sigmoid ? 0.f : -INFINITY, sum = 0.f;
    float o[2 * N][4];
#pragma unroll
    for (int j = 0; j < 2 * N; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
    // A tile is blocks of 64 columns, [KT rows x 128 bytes] with the 16-byte pieces of row r at place (piece ^ (r & 7)).  Columns
    // 16 (w + 8 i) .. + 15 lie in block w / 4 + 2 i, pieces 2 (w % 4) and the next one, for the keys as for the values.
    const int block0 = (w >> 2) * KT * 128, mine = 2 * (w & 3);
    const int k_at = block0 + ((l & 7) + 8 * (l >> 4)) * 128 + (((mine + ((l >> 3) & 1)) ^ (l & 7)) << 4);       // ldmatrix, two key groups of 8
    const int v_at = block0 + ((l & 7) + 8 * ((l >> 3) & 1)) * 128 + (((mine + (l >> 4)) ^ (l & 7)) << 4);      // transposing, two strips of 8
    const bf16* q_at = Q + ((l & 7) + 8 * ((l >> 3) & 1)) * L.q_ld + 16 * w + 8 * (l >> 4);
    float* s_at = S + (w * ROWS + g) * (KT + 4) + 2 * q;
    const float* x_at = S + srow * (KT + 4) + sk0;
    const bool scoring = w < bufs;

    // partial scores of tile t; false when its data did not arrive in time
    auto scores = [&](int t, int st, uint32_t phase) -> bool {
        const bool ok = fatc::mbar_wait_suspend(&full[st], phase, &abort_flag, err, 0xa100 | st);
        unsigned char* tile = smem + st * L.stage;
        const int valid = nk - t * KT;
        if (valid < KT) {                                    // (the request's last tile) values that meet a probability of zero
            const int blocks = (a.dv + 63) / 64;
            for (int i = threadIdx.x; i < blocks * (KT - valid) * 8; i += THREADS) {
                const int rows = KT - valid, c = i % 8, j = i / 8 % rows, blk = i / 8 / rows;
                *reinterpret_cast<uint4*>(tile + L.v + (blk * KT + valid + j) * 128 + c * 16) = make_uint4(0, 0, 0, 0);
            }
        }
        if (!scoring) return ok;
        float s[2 * KE][4];
#pragma unroll
        for (int e = 0; e < 2 * KE; ++e) s[e][0] = s[e][1] = s[e][2] = s[e][3] = 0.f;
#pragma unroll
        for (int i = 0; i < N; ++i) {
            if (i == 0 || (w + WARPS * i) * 16 < a.dk) {
                uint32_t qa[4], kb[4];
                ldsm_x4(qa, q_at + 128 * i);
#pragma unroll
                for (int e = 0; e < KE; ++e) {
                    ldsm_x4(kb, tile + k_at + 2 * i * KT * 128 + e * 2048);
                    mma16816(s[2 * e], qa, kb[0], kb[1]);
                    mma16816(s[2 * e + 1], qa, kb[2], kb[3]);
                }
            }
        }
#pragma unroll
        for (int e = 0; e < 2 * KE; ++e) {
            *reinterpret_cast<float2*>(s_at + 8 * e) = make_float2(s[e][0], s[e][1]);
            *reinterpret_cast<float2*>(s_at + 8 * e + 8 * (KT + 4)) = make_float2(s[e][2], s[e][3]);
        }
        return ok;
    };

    int st = 0;
    uint32_t phase = 0;
    bool go = true;
    if (t_beg < t_end) go = __syncthreads_and(scores(t_beg, 0, 0));
    for (int t = t_beg; go && t < t_end; ++t) {
        {
            float x[KPT];
#pragma unroll
            for (int i = 0; i < KPT; ++i) x[i] = 0.f;
#pragma unroll
            for (int r = 0; r < WARPS; ++r)
                if (r < bufs) {
#pragma unroll
                    for (int i = 0; i < KPT; i += 2) {
                        const float2 f = *reinterpret_cast<const float2*>(x_at + r * ROWS * (KT + 4) + i);
                        x[i] += f.x;
                        x[i + 1] += f.y;
                    }
                }
            if (sigmoid) {
#pragma unroll
                for (int i = 0; i < KPT; i += 2) {
                    const int key = t * KT + sk0 + i;
                    x[i] = key >= lo && key < nk ? rcp(1.f + ex2(-(x[i] * sc + head_bias))) : 0.f;
                    x[i + 1] = key + 1 >= lo && key + 1 < nk ? rcp(1.f + ex2(-(x[i + 1] * sc + head_bias))) : 0.f;
                    *reinterpret_cast<__nv_bfloat162*>(P + srow * (KT + 8) + sk0 + i) = __floats2bfloat162_rn(x[i], x[i + 1]);
                }
                if (sk0 == 0) ML[2 * ROWS + srow] = 1.f;
            } else {
                float mx = m;
                if (t * KT >= lo && (t + 1) * KT <= nk) {
#pragma unroll
                    for (int i = 0; i < KPT; ++i) x[i] *= sc;
                } else {
#pragma unroll
                    for (int i = 0; i < KPT; ++i) {
                        const int key = t * KT + sk0 + i;
                        x[i] = key >= lo && key < nk ? x[i] * sc : -INFINITY;
                    }
                }
#pragma unroll
                for (int i = 0; i < KPT; ++i) mx = fmaxf(mx, x[i]);
#pragma unroll
                for (int d = 1; d < TPR; d <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
                const float corr = m == -INFINITY ? 0.f : ex2(m - mx);       // a tile of [lo, nk) has a visible key: mx is finite
                sum *= corr;                                                 // this thread's keys only, added up at the end
#pragma unroll
                for (int i = 0; i < KPT; i += 2) {
                    x[i] = ex2(x[i] - mx);
                    x[i + 1] = ex2(x[i + 1] - mx);
                    sum += x[i] + x[i + 1];
                    *reinterpret_cast<__nv_bfloat162*>(P + srow * (KT + 8) + sk0 + i) = __floats2bfloat162_rn(x[i], x[i + 1]);
                }
                m = mx;
                if (sk0 == 0) ML[2 * ROWS + srow] = corr;
            }
        }
        __syncthreads();
        {
            const float c0 = ML[2 * ROWS + g], c1 = ML[2 * ROWS + g + 8];
#pragma unroll
            for (int j = 0; j < 2 * N; ++j) {
                o[j][0] *= c0; o[j][1] *= c0;
                o[j][2] *= c1; o[j][3] *= c1;
            }
        }
        const unsigned char* vt = smem + st * L.stage + L.v + v_at;
        uint32_t pf[KE][4];
#pragma unroll
        for (int e = 0; e < KE; ++e) load_a(pf[e], P, KT + 8, 0, 16 * e);
#pragma unroll
        for (int j = 0; j < N; ++j) {
            if ((w + WARPS * j) * 16 < a.dv) {
#pragma unroll
                for (int e = 0; e < KE; ++e) {
                    uint32_t vb[4];
                    ldsm_x4_t(vb, vt + 2 * j * KT * 128 + e * 2048);
                    mma16816(o[2 * j], pf[e], vb[0], vb[1]);
                    mma16816(o[2 * j + 1], pf[e], vb[2], vb[3]);
                }
            }
        }
        const int now = st;
        if (++st == stages) {
            st = 0;
            phase ^= 1;
        }
        go = __syncthreads_and(t + 1 < t_end ? scores(t + 1, st, phase) : true);
        if (threadIdx.x == 0 && go && t + stages < t_end) load(t + stages, now);
    }
    __syncthreads();
#pragma unroll
    for (int d = 1; d < TPR; d <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, d);
    // join the cluster: every CTA finishes some of the heads
    float* O = reinterpret_cast<float*>(smem);               // [ROWS][dv + 4]
    const int o_ld = a.dv + 4;
#pragma unroll
    for (int j = 0; j < N; ++j) {
        const int n0 = (w + WARPS * j) * 16;
        if (n0 < a.dv) {
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                float* p = O + g * o_ld + n0 + 8 * e + 2 * q;
                *reinterpret_cast<float2*>(p) = make_float2(o[2 * j + e][0], o[2 * j + e][1]);
                *reinterpret_cast<float2*>(p + 8 * o_ld) = make_float2(o[2 * j + e][2], o[2 * j + e][3]);
            }
        }
    }
    if (sk0 == 0) {
        ML[srow] = m;
        ML[ROWS + srow] = sum;
    }
    auto cluster = cg::this_cluster();
    cluster.sync();
    for (int i = threadIdx.x; i < splits * ROWS; i += THREADS) {
        const float* ml = cluster.map_shared_rank(ML, i / ROWS);
        part[0][i / ROWS][i % ROWS] = ml[i % ROWS];
        part[1][i / ROWS][i % ROWS] = ml[ROWS + i % ROWS];
    }
    __syncthreads();
    const int vp = a.dv / 4, wpr = vp <= 32 ? 1 : vp <= 64 ? 2 : 4;      // warps per row
    for (int h = split + splits * (w / wpr); h < nh; h += splits * (WARPS / wpr)) {
        float mx = -INFINITY;
        for (int r = 0; r < splits; ++r) mx = fmaxf(mx, part[0][r][h]);
        for (int d = (w % wpr) * 32 + l; d < vp; d += wpr * 32) {
            float ls = 0.f;
            float4 os = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
            for (int r = 0; r < splits; ++r) {
                const float f = part[0][r][h] == -INFINITY ? 0.f : ex2(part[0][r][h] - mx);
                const float4 x = *reinterpret_cast<const float4*>(cluster.map_shared_rank(O, r) + h * o_ld + 4 * d);
                ls += part[1][r][h] * f;
                os.x += x.x * f; os.y += x.y * f; os.z += x.z * f; os.w += x.w * f;
            }
            const float inv = sigmoid ? a.mul : 1.f / ls;
            __nv_bfloat162 y[2] = {__floats2bfloat162_rn(os.x * inv, os.y * inv), __floats2bfloat162_rn(os.z * inv, os.w * inv)};
            *reinterpret_cast<uint2*>((bf16*)a.out + (long long)b * a.ldo + (long long)(h0 + h) * a.dv + 4 * d) = *reinterpret_cast<uint2*>(y);
        }
    }
    cluster.sync();                                          // nobody leaves while its shared memory is read
}

template <int KT, int N, bool SHARED>
static int launch(const Step& a, int rows, int splits, int* err, cudaStream_t st) {
    // as many stages as leave room for two CTAs per SM, or for one where there is no second one
    constexpr int STATIC = 128 + 2 * MAX_SPLITS * ROWS * 4, ROOM = 227 * 1024 - STATIC, HALF = 227 * 512 - STATIC - 1024;
    static int sms = 0;
    if (sms == 0) {
        int dev = 0;
        if (cudaGetDevice(&dev) != cudaSuccess || cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess) sms = 148;
    }
    const dim3 grid(splits, a.G * ((a.H / a.G + ROWS - 1) / ROWS), a.n);
    // (wide clusters do not fill every SM at one CTA each)
    const long long ctas = (long long)grid.x * grid.y * grid.z;
    const bool alone = ctas * (splits > 4 ? 2 : 1) <= sms;
    const int room = !alone && Layout(KT, a.dk, a.dv, SHARED, 2).total <= HALF ? HALF : ROOM;
    int stages = MAX_STAGES;
    while (stages > 2 && Layout(KT, a.dk, a.dv, SHARED, stages).total > room) --stages;
    const int smem = Layout(KT, a.dk, a.dv, SHARED, stages).total;
    if (smem > ROOM) return -2;
    CUtensorMap mk, mv;
    int rc = fatc::make_map_4d(&mk, a.c.k, 1, rows, a.G, a.dk, (long long)rows * a.G * a.dk, (long long)a.G * a.dk, a.dk, KT);
    if (rc == 0) rc = SHARED ? (mv = mk, 0) : fatc::make_map_4d(&mv, a.c.v, 1, rows, a.G, a.dv, (long long)rows * a.G * a.dv, (long long)a.G * a.dv, a.dv, KT);
    if (rc) return rc;
    auto kern = packed_attn_step_kernel<KT, N, SHARED>;
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e == cudaSuccess && splits > 8) e = cudaFuncSetAttribute(kern, cudaFuncAttributeNonPortableClusterSizeAllowed, 1);
    if (e != cudaSuccess) return (int)e;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
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
    return (int)cudaLaunchKernelEx(&cfg, kern, mk, mv, a, stages, err);
}

template <bool SHARED>
static int by_width(const Step& a, int rows, int splits, int* err, cudaStream_t st) {
    const int wide = a.dk > a.dv ? a.dk : a.dv;
    if (wide <= 128) return launch<64, 1, SHARED>(a, rows, splits, err, st);
    if (wide <= 256) return launch<32, 2, SHARED>(a, rows, splits, err, st);
    return launch<32, 4, SHARED>(a, rows, splits, err, st);
}

}  // namespace pas
}  // namespace lmoe

using namespace lmoe;

// bf16, head sizes multiples of 16 up to 512, 16-byte aligned bases, pitches multiples of 8; a.c.v == a.c.k (and dv ==
// dk): the rows are key and value at once.  rows: all rows of the cache buffers.  splits: 1, 2, 4, 8 or 16 CTAs per (request, heads).
// Slots, positions and the page table must have been on the device before the kernel that precedes this one in the stream was
// launched; that kernel stores the new token.  err: status word of the bounded waits.  Returns -2 when the head sizes do not fit
// shared memory.
LMOE_API int lmoe_packed_attn_step(const pa::Step* ap, int rows, int splits, int* err, cudaStream_t st) {
    const pa::Step& a = *ap;
    if (a.n <= 0 || a.G <= 0 || a.H <= 0 || a.H % a.G || a.dk <= 0 || a.dv <= 0 || a.dk % 16 || a.dv % 16 || a.dk > 512 || a.dv > 512 || a.ldq % 8 || a.ldo % 8 ||
        rows <= 0 || (a.bias == nullptr && !(a.scale > 0.f)) || a.cross || (a.c.table == nullptr && a.c.cap <= 0) ||
        ((reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(a.c.k) | reinterpret_cast<uintptr_t>(a.c.v) |
          reinterpret_cast<uintptr_t>(a.out)) & 15) ||
        (splits != 1 && splits != 2 && splits != 4 && splits != 8 && splits != 16))
        return -1;
    if (a.c.v == a.c.k) return a.dk != a.dv ? -1 : pas::by_width<true>(a, rows, splits, err, st);
    return pas::by_width<false>(a, rows, splits, err, st);
}
