// Softmax attention inside fixed chunks of the sequence (position i sees j <= i when i / size == j / size), with soft-capped
// scores, a learned bias per distance and head, and an output gate:
//     s = cap * tanh(q . k * scale / cap) + bias[h][i - j],   o = mul * sigmoid(gate) * (softmax(s) v)
// Queries, keys, values and gates are column ranges of one projection output [tokens, ldz]; `gain` is the one-number gain
// of the norm before that projection, applied here (squared on the scores).  Requests of a batch are packed: request r's
// tokens are consecutive rows, and all kernels work on rows, so prompts of any lengths share a launch.
//
// A chunk never looks outside itself, so the cache of a request is one chunk: row `position % size`, overwritten when the
// next chunk begins.
//
//   chunk_attn_rows_kernel   prompts, any head sizes, bf16 or fp32 (all arithmetic fp32): tiles of 32 queries x 32 keys,
//                            online softmax.  Keys of the chunk that precede this call come from the cache.  The bf16 fast path for
//                            prompts is chunk_attn_tc.cu.
//   chunk_attn_step_kernel   one token per request, any head sizes, bf16 or fp32 (bf16 fast path: chunk_attn_step.cu): a cluster of CTAs splits the keys of (request, kv head), the partial
//                            softmaxes meet in distributed shared memory; the new key and value are read from the projection and
//                            stored into the cache on the way; the gate is applied in the same kernel
//   chunk_store_kernel       keys / values of a prompt's last chunk -> cache
// Compiled without fast-math.
#include <cooperative_groups.h>

#include "chunk_attn.cuh"
#include "common.cuh"
#include "mma_utils.cuh"

namespace lmoe {
namespace ca {
namespace cg = cooperative_groups;

__device__ __forceinline__ float capped(float s, float cap) { return cap > 0.f ? cap * tanhf(s / cap) : s; }

// ---------------------------------------------------------------------------------------------------- prompts, any size
constexpr int RQ = 32, RK = 32, RT = 128;

template <typename T>
__global__ void __launch_bounds__(RT) chunk_attn_rows_kernel(Args a) {
    extern __shared__ float sm[];
    const int dk = a.dk, dv = a.dv, ldk = dk + 1;
    float* Q = sm;                       // [RQ][dk + 1]
    float* K = Q + RQ * ldk;             // [RK][dk + 1]
    float* V = K + RK * ldk;             // [RK][dv]
    float* O = V + RK * dv;              // [RQ][dv]
    float* S = O + RQ * dv;              // [RQ][RK + 1]
    const int* it = a.items + (long long)blockIdx.x * I_N;
    const int row0 = it[I_ROW], nq = it[I_NQ], c0 = it[I_C0], fresh0 = it[I_FRESH0], slot = it[I_SLOT];
    const int h = blockIdx.y, hk = h / (a.H / a.G);
    const T* z = (const T*)a.z;
    const float gain = *a.gain, sc = a.scale * gain * gain;
    for (int i = threadIdx.x; i < RQ * dk; i += RT) {
        const int r = i / dk, d = i % dk;
        Q[r * ldk + d] = r < nq ? to_f(z[(row0 + r) * a.ldz + a.zq + h * dk + d]) : 0.f;
    }
    for (int i = threadIdx.x; i < RQ * dv; i += RT) O[i] = 0.f;
    const int r = threadIdx.x >> 2, part = threadIdx.x & 3;            // four threads per query row
    const float* bias = a.lut + (long long)h * a.nlut;
    float m = -INFINITY, l = 0.f;
    const int nk = c0 + nq;                                            // keys 0 .. nk - 1 of the chunk
    for (int k0 = 0; k0 < nk; k0 += RK) {
        __syncthreads();
        for (int i = threadIdx.x; i < RK * dk; i += RT) {
            const int j = i / dk, d = i % dk, key = k0 + j;
            float v = 0.f;
            if (key < nk)
                v = key >= fresh0 ? to_f(z[(row0 - c0 + key) * a.ldz + a.zk + hk * dk + d])
                                  : to_f(((const T*)a.kc)[(((long long)slot * a.cap_rows + key) * a.G + hk) * a.dkp + d]);
            K[j * ldk + d] = v;
        }
        for (int i = threadIdx.x; i < RK * dv; i += RT) {
            const int j = i / dv, d = i % dv, key = k0 + j;
            float v = 0.f;
            if (key < nk)
                v = key >= fresh0 ? to_f(z[(row0 - c0 + key) * a.ldz + a.zv + hk * dv + d])
                                  : to_f(((const T*)a.vc)[(((long long)slot * a.cap_rows + key) * a.G + hk) * a.dvp + d]);
            V[i] = v;
        }
        __syncthreads();
        float s[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) s[e] = 0.f;
        for (int d = 0; d < dk; ++d) {
            const float q = Q[r * ldk + d];
#pragma unroll
            for (int e = 0; e < 8; ++e) s[e] += q * K[(part + 4 * e) * ldk + d];
        }
        float mx = m;
#pragma unroll
        for (int e = 0; e < 8; ++e) {
            const int dist = c0 + r - (k0 + part + 4 * e);
            s[e] = dist >= 0 ? capped(s[e] * sc, a.cap) + bias[min(dist, a.nlut - 1)] : -INFINITY;
            mx = fmaxf(mx, s[e]);
        }
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        const float corr = m == -INFINITY ? 0.f : expf(m - mx);       // key 0 is visible to every query: mx is finite
        float ps = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) {
            const float p = expf(s[e] - mx);
            S[r * (RK + 1) + part + 4 * e] = p;
            ps += p;
        }
        ps += __shfl_xor_sync(0xffffffffu, ps, 1);
        ps += __shfl_xor_sync(0xffffffffu, ps, 2);
        l = l * corr + ps;
        m = mx;
        __syncwarp();
        for (int d = part; d < dv; d += 4) {
            float o = O[r * dv + d] * corr;
            for (int j = 0; j < RK; ++j) o += S[r * (RK + 1) + j] * V[j * dv + d];
            O[r * dv + d] = o;
        }
        __syncwarp();
    }
    if (r < nq) {
        T* out = (T*)a.out + (row0 + r) * a.ldo + h * dv;
        const T* g = z + (row0 + r) * a.ldz + a.zg + h * dv;
        const float w = a.mul * gain / l;
        for (int d = part; d < dv; d += 4) {
            const float gate = 1.f / (1.f + expf(-gain * to_f(g[d])));
            out[d] = from_f<T>(O[r * dv + d] * w * gate);
        }
    }
}

// --------------------------------------------------------------------------------------------------------- one token
constexpr int ST = 128, HT = 8;          // threads, query heads handled together

template <typename T>
struct StepSmem {                        // offsets (in bytes) inside the dynamic shared memory
    int kt, k_ld, v_ld;                  // keys per tile, padded row lengths (elements)
    int k, v, q, p, acc, ml, total;
    __host__ __device__ StepSmem(int kt_, int dk, int dv) : kt(kt_) {
        constexpr int E = 16 / (int)sizeof(T);
        k_ld = (dk + E - 1) / E * E + E;               // rows stay 16-byte aligned and fall into different banks
        v_ld = (dv + E - 1) / E * E;
        k = 0;
        v = k + 2 * kt * k_ld * (int)sizeof(T);
        q = v + 2 * kt * v_ld * (int)sizeof(T);
        p = q + HT * ((dk + 7) / 8 * 8) * 4;
        acc = p + HT * kt * 4;
        ml = acc + HT * ((dv + 3) / 4 * 4) * 4;
        total = ml + 3 * HT * 4;
    }
};

// Stage keys [k0, k0 + kt) of (request, kv head) into buffer `buf`: cache rows, except key `cur`, which is the new token's
// row of the projection.  vec: rows are whole 16-byte pieces.
template <typename T>
__device__ __forceinline__ void step_load(const Args& a, const StepSmem<T>& L, unsigned char* sm, int buf, int k0, int k_hi, int cur,
                                          int hk, long long cache_row0, const T* zrow, int vec) {
    T* Ks = reinterpret_cast<T*>(sm + L.k) + buf * L.kt * L.k_ld;
    T* Vs = reinterpret_cast<T*>(sm + L.v) + buf * L.kt * L.v_ld;
    const T* kc = (const T*)a.kc;
    const T* vc = (const T*)a.vc;
    if (vec) {
        constexpr int E = 16 / (int)sizeof(T);
        const int kp = a.dk / E, vp = a.dv / E;
        for (int i = threadIdx.x; i < L.kt * kp; i += ST) {
            const int j = i / kp, c = (i % kp) * E, key = k0 + j;
            const T* src = key == cur ? zrow + a.zk + hk * a.dk + c : kc + ((cache_row0 + key) * a.G + hk) * a.dkp + c;
            cp_async16(Ks + j * L.k_ld + c, key < k_hi ? src : kc, key < k_hi);
        }
        for (int i = threadIdx.x; i < L.kt * vp; i += ST) {
            const int j = i / vp, c = (i % vp) * E, key = k0 + j;
            const T* src = key == cur ? zrow + a.zv + hk * a.dv + c : vc + ((cache_row0 + key) * a.G + hk) * a.dvp + c;
            cp_async16(Vs + j * L.v_ld + c, key < k_hi ? src : vc, key < k_hi);
        }
    } else {
        for (int i = threadIdx.x; i < L.kt * a.dk; i += ST) {
            const int j = i / a.dk, c = i % a.dk, key = k0 + j;
            T v = from_f<T>(0.f);
            if (key < k_hi) v = key == cur ? zrow[a.zk + hk * a.dk + c] : kc[((cache_row0 + key) * a.G + hk) * a.dkp + c];
            Ks[j * L.k_ld + c] = v;
        }
        for (int i = threadIdx.x; i < L.kt * a.dv; i += ST) {
            const int j = i / a.dv, c = i % a.dv, key = k0 + j;
            T v = from_f<T>(0.f);
            if (key < k_hi) v = key == cur ? zrow[a.zv + hk * a.dv + c] : vc[((cache_row0 + key) * a.G + hk) * a.dvp + c];
            Vs[j * L.v_ld + c] = v;
        }
    }
    cp_async_commit();
}

// grid (splits, G * head tiles, B), cluster (splits, 1, 1)
template <typename T>
__global__ void __launch_bounds__(ST) chunk_attn_step_kernel(Args a, int kt, int vec) {
    pdl_trigger();
    extern __shared__ __align__(16) unsigned char smem[];
    const StepSmem<T> L(kt, a.dk, a.dv);
    float* Q = reinterpret_cast<float*>(smem + L.q);
    float* P = reinterpret_cast<float*>(smem + L.p);
    float* ACC = reinterpret_cast<float*>(smem + L.acc);
    float* ML = reinterpret_cast<float*>(smem + L.ml);       // [HT] max, [HT] sum, [HT] correction of the current tile
    const int qp = (a.dk + 7) / 8 * 8, ap = (a.dv + 3) / 4 * 4;
    const int splits = gridDim.x, split = blockIdx.x, b = blockIdx.z;
    const int qpg = a.H / a.G, tiles = (qpg + HT - 1) / HT;
    const int hk = blockIdx.y / tiles, h0 = hk * qpg + (blockIdx.y % tiles) * HT;
    const int nh = min(HT, hk * qpg + qpg - h0);
    const int slot = a.slots[b], cur = a.pos[b] % a.size;    // the new token's place in its chunk
    const int nk = cur + 1;
    const int per = ((nk + splits - 1) / splits + kt - 1) / kt * kt;
    const int k_lo = split * per, k_hi = min(nk, k_lo + per);
    const T* zrow = (const T*)a.z + (long long)b * a.ldz;
    const long long cache_row0 = (long long)slot * a.cap_rows;
    const float gain = *a.gain, sc = a.scale * gain * gain;
    const int w = threadIdx.x >> 5, lane = threadIdx.x & 31;

    if (k_lo < k_hi) step_load<T>(a, L, smem, 0, k_lo, k_hi, cur, hk, cache_row0, zrow, vec);
    for (int i = threadIdx.x; i < HT * qp; i += ST) {
        const int h = i / qp, d = i % qp;
        Q[i] = (h < nh && d < a.dk) ? to_f(zrow[a.zq + (h0 + h) * a.dk + d]) * sc : 0.f;
    }
    for (int i = threadIdx.x; i < HT * ap; i += ST) ACC[i] = 0.f;
    if (threadIdx.x < HT) {
        ML[threadIdx.x] = -INFINITY;
        ML[HT + threadIdx.x] = 0.f;
    }
    // the new key and value enter the cache (read from the projection above, so nothing here depends on the store)
    if (h0 == hk * qpg && cur >= k_lo && cur < k_hi) {
        T* kd = (T*)a.kc + ((cache_row0 + cur) * a.G + hk) * a.dkp;
        T* vd = (T*)a.vc + ((cache_row0 + cur) * a.G + hk) * a.dvp;
        for (int d = threadIdx.x; d < a.dk; d += ST) kd[d] = zrow[a.zk + hk * a.dk + d];
        for (int d = threadIdx.x; d < a.dv; d += ST) vd[d] = zrow[a.zv + hk * a.dv + d];
    }
    constexpr int E = 16 / (int)sizeof(T);
    int buf = 0;
    for (int k0 = k_lo; k0 < k_hi; k0 += kt, buf ^= 1) {
        if (k0 + kt < k_hi) step_load<T>(a, L, smem, buf ^ 1, k0 + kt, k_hi, cur, hk, cache_row0, zrow, vec);
        else cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const T* Ks = reinterpret_cast<const T*>(smem + L.k) + buf * kt * L.k_ld;
        const T* Vs = reinterpret_cast<const T*>(smem + L.v) + buf * kt * L.v_ld;
        // scores: a thread owns one key of the tile for every (ST / kt)-th head
        {
            const int j = threadIdx.x % kt, hg = threadIdx.x / kt, nhg = ST / kt, key = k0 + j;
            const T* kr = Ks + j * L.k_ld;
            for (int hb = hg; hb < nh; hb += 4 * nhg) {               // four heads at a time
                float s[4] = {0.f, 0.f, 0.f, 0.f};
                int hx[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) hx[e] = min(hb + e * nhg, HT - 1) * qp;
                int d = 0;
                for (; d + E <= a.dk; d += E) {
                    Vec<T> kv;
                    kv.load(kr + d);
#pragma unroll
                    for (int i = 0; i < E; ++i) {
                        const float kf = kv.get(i);
#pragma unroll
                        for (int e = 0; e < 4; ++e) s[e] += kf * Q[hx[e] + d + i];
                    }
                }
                for (; d < a.dk; ++d) {
                    const float kf = to_f(kr[d]);
#pragma unroll
                    for (int e = 0; e < 4; ++e) s[e] += kf * Q[hx[e] + d];
                }
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int h = hb + e * nhg;
                    if (h < nh)
                        P[h * kt + j] = key < k_hi ? capped(s[e], a.cap) + a.lut[(long long)(h0 + h) * a.nlut + min(cur - key, a.nlut - 1)]
                                                   : -INFINITY;
                }
            }
        }
        __syncthreads();
        // running maximum and sum: one warp per head
        for (int h = w; h < nh; h += ST / 32) {
            const float m_old = ML[h];
            float mx = m_old;
            for (int j = lane; j < kt; j += 32) mx = fmaxf(mx, P[h * kt + j]);
            mx = warp_max(mx);
            float ps = 0.f;
            for (int j = lane; j < kt; j += 32) {
                const float p = expf(P[h * kt + j] - mx);
                P[h * kt + j] = p;
                ps += p;
            }
            ps = warp_sum(ps);
            __syncwarp();
            if (lane == 0) {
                const float corr = m_old == -INFINITY ? 0.f : expf(m_old - mx);
                ML[2 * HT + h] = corr;
                ML[HT + h] = ML[HT + h] * corr + ps;
                ML[h] = mx;
            }
        }
        __syncthreads();
        // values: a thread owns a column for all heads
        for (int d = threadIdx.x; d < a.dv; d += ST) {
            float o[HT];
#pragma unroll
            for (int h = 0; h < HT; ++h) o[h] = h < nh ? ACC[h * ap + d] * ML[2 * HT + h] : 0.f;
            for (int j = 0; j < kt; j += 4) {
                float v[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) v[i] = to_f(Vs[(j + i) * L.v_ld + d]);
#pragma unroll
                for (int h = 0; h < HT; ++h) {
                    if (h < nh) {
                        const float4 p = *reinterpret_cast<const float4*>(P + h * kt + j);
                        o[h] += p.x * v[0] + p.y * v[1] + p.z * v[2] + p.w * v[3];
                    }
                }
            }
#pragma unroll
            for (int h = 0; h < HT; ++h)
                if (h < nh) ACC[h * ap + d] = o[h];
        }
        __syncthreads();
    }
    cp_async_wait<0>();
    __syncthreads();
    // join the splits: every CTA of the cluster finishes a slice of the (head, column) pairs
    auto cluster = cg::this_cluster();
    cluster.sync();
    for (int i = split * ST + threadIdx.x; i < nh * a.dv; i += splits * ST) {
        const int h = i / a.dv, d = i % a.dv;
        float m = -INFINITY;
        for (int s = 0; s < splits; ++s) m = fmaxf(m, cluster.map_shared_rank(ML, s)[h]);
        float l = 0.f, o = 0.f;
        for (int s = 0; s < splits; ++s) {
            const float* ml = cluster.map_shared_rank(ML, s);
            const float f = ml[h] == -INFINITY ? 0.f : expf(ml[h] - m);
            l += ml[HT + h] * f;
            o += cluster.map_shared_rank(ACC, s)[h * ap + d] * f;
        }
        const int col = (h0 + h) * a.dv + d;
        const float gate = 1.f / (1.f + expf(-gain * to_f(zrow[a.zg + col])));
        ((T*)a.out)[(long long)b * a.ldo + col] = from_f<T>(o / l * (a.mul * gain) * gate);
    }
    cluster.sync();                                          // nobody leaves while its shared memory is read
}

// ------------------------------------------------------------------------------------------------------ prompt -> cache
template <typename T>
__global__ void chunk_store_kernel(Args a) {
    const int row = blockIdx.x, p = a.pos[row];
    if (p / a.size != a.ends[row] / a.size) return;          // only the chunk that the next token belongs to is kept
    const T* zr = (const T*)a.z + (long long)row * a.ldz;
    const long long r = ((long long)a.slots[row] * a.cap_rows + p % a.size) * a.G;
    for (int i = threadIdx.x; i < a.G * a.dk; i += blockDim.x) ((T*)a.kc)[(r + i / a.dk) * a.dkp + i % a.dk] = zr[a.zk + i];
    for (int i = threadIdx.x; i < a.G * a.dv; i += blockDim.x) ((T*)a.vc)[(r + i / a.dv) * a.dvp + i % a.dv] = zr[a.zv + i];
}

template <typename T>
static int launch_rows(const Args& a, cudaStream_t st) {
    const size_t smem = sizeof(float) * ((RQ + RK) * (size_t)(a.dk + 1) + (RK + RQ) * (size_t)a.dv + RQ * (RK + 1));
    if (smem > 227 * 1024) return -2;                        // head sizes beyond about 400
    cudaError_t e = cudaFuncSetAttribute(chunk_attn_rows_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    chunk_attn_rows_kernel<T><<<dim3(a.n, a.H), RT, smem, st>>>(a);
    return (int)cudaGetLastError();
}

template <typename T>
static int launch_step(const Args& a, int splits, cudaStream_t st) {
    int kt = 64;
    while (kt > 16 && StepSmem<T>(kt, a.dk, a.dv).total > 100 * 1024) kt /= 2;
    const int smem = StepSmem<T>(kt, a.dk, a.dv).total;
    if (smem > 227 * 1024) return -2;
    constexpr int E = 16 / (int)sizeof(T);
    const int vec = a.dk % E == 0 && a.dv % E == 0 && a.ldz % E == 0 && a.zk % E == 0 && a.zv % E == 0 && a.dkp % E == 0 && a.dvp % E == 0;
    cudaError_t e = cudaFuncSetAttribute(chunk_attn_step_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return (int)e;
    const int qpg = a.H / a.G;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(splits, a.G * ((qpg + HT - 1) / HT), a.n);
    cfg.blockDim = dim3(ST);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = splits;
    attr[0].val.clusterDim.y = 1;
    attr[0].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    return (int)cudaLaunchKernelEx(&cfg, chunk_attn_step_kernel<T>, a, kt, vec);
}

static bool sane(const Args& a) {
    return a.n > 0 && a.H > 0 && a.G > 0 && a.H % a.G == 0 && a.dk > 0 && a.dv > 0 && a.dkp >= a.dk && a.dvp >= a.dv && a.size > 0 &&
           a.nlut > 0;
}

}  // namespace ca
}  // namespace lmoe

using namespace lmoe;

// dt: 1 bf16, 0 fp32.  items [n, 8] int32: packed row of the first query, queries (<= 32), its place in its chunk, place of the
// first key that is in this call (earlier ones are in the cache), cache slot.
LMOE_API int lmoe_chunk_attn_rows(const ca::Args* ap, int dt, cudaStream_t st) {
    if (!ca::sane(*ap)) return -1;
    return dt ? ca::launch_rows<bf16>(*ap, st) : ca::launch_rows<float>(*ap, st);
}

// splits: 1, 2, 4 or 8 CTAs per (request, kv head)
LMOE_API int lmoe_chunk_attn_step(const ca::Args* ap, int splits, int dt, cudaStream_t st) {
    if (!ca::sane(*ap) || (splits != 1 && splits != 2 && splits != 4 && splits != 8)) return -1;
    return dt ? ca::launch_step<bf16>(*ap, splits, st) : ca::launch_step<float>(*ap, splits, st);
}

LMOE_API int lmoe_chunk_store(const ca::Args* ap, int dt, cudaStream_t st) {
    if (!ca::sane(*ap)) return -1;
    if (dt) ca::chunk_store_kernel<bf16><<<ap->n, 128, 0, st>>>(*ap);
    else ca::chunk_store_kernel<float><<<ap->n, 128, 0, st>>>(*ap);
    return (int)cudaGetLastError();
}
