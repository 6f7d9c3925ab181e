// Packed-row attention (softmax or sigmoid weights) for any head size, bf16 or fp32 (arithmetic in fp32), and the row kernels around it:
//   packed_attn_rows_kernel   prompts (mathematics and work items: packed_attn_tc.cu, the bf16 fast path): tiles of TQ queries x TQ
//                             keys, online softmax
//   packed_attn_step_kernel   one token per request from the cache (bf16 fast path: packed_attn_step.cu)
//   qk_norm_rope_kernel       RMS norm of all query rows of a projection and of all key rows, before the heads are split, then
//                             interleaved rotary positions, in place; the new keys and values enter the cache
//   rotary_rows_kernel        cos and sin of every row's angles, for all layers that rotate alike
//   head_norm_rope_kernel     RMS norm of every query, key and value head, rotary positions in either pairing, values mixed with another
//                             layer's, in place; the new keys and values enter the cache
//   head_mix_kernel           talking heads: the outputs of every head's weights over every value head -> the heads' outputs
//   latent_norm_kernel        RMS norm of a latent projection into a matrix of its own and into the cache
//   gather_rows_kernel        rows of a matrix and of a cache -> rows of a buffer (a prompt that goes on from a cache)
//   gate_rows_kernel          o *= sigmoid(g)
// Compiled without fast-math: the fp32 instantiations serve models in true 32-bit.
#include "common.cuh"
#include "packed_attn.cuh"

namespace lmoe {
namespace pag {
using pa::Cache;
using pa::Prompt;
using pa::Step;

// ------------------------------------------------------------------------------------------------------------------ prompts
// TQ queries (32 or 16), four threads per query
template <typename T, int TQ>
__global__ void __launch_bounds__(TQ * 4) packed_attn_rows_kernel(Prompt a) {
    constexpr int TK = TQ, NT = TQ * 4, KP = TK / 4;
    extern __shared__ float sm[];
    const int dk = a.dk, dv = a.dv, ldk = dk + 1;
    float* Q = sm;                       // [TQ][dk + 1]
    float* K = Q + TQ * ldk;             // [TK][dk + 1]
    float* V = K + TK * ldk;             // [TK][dv]
    float* O = V + TK * dv;              // [TQ][dv]
    float* S = O + TQ * dv;              // [TQ][TK + 1]
    const int* it = a.items + (long long)blockIdx.x * pa::I_N;
    const int row0 = it[pa::I_ROW], nq = it[pa::I_NQ], c0 = it[pa::I_C0], krow = it[pa::I_KROW];
    const int h = blockIdx.y, hk = h / (a.H / a.G);
    const int hv = a.cross ? blockIdx.z : hk, ho = a.cross ? h * a.G + hv : h;      // value head, head of the output
    for (int i = threadIdx.x; i < TQ * dk; i += NT) {
        const int r = i / dk, d = i % dk;
        Q[r * ldk + d] = r < nq ? to_f(((const T*)a.q)[(row0 + r) * a.ldq + h * dk + d]) : 0.f;
    }
    for (int i = threadIdx.x; i < TQ * dv; i += NT) O[i] = 0.f;
    const int r = threadIdx.x >> 2, part = threadIdx.x & 3;
    const int qi = c0 + min(r, nq - 1);  // rows beyond the item repeat its last query
    float m = -INFINITY, l = 0.f;
    const int k_beg = a.window > 0 ? max(0, c0 - a.window + 1) : 0, k_end = c0 + nq;
    for (int k0 = k_beg; k0 < k_end; k0 += TK) {
        __syncthreads();
        for (int i = threadIdx.x; i < TK * dk; i += NT) {
            const int j = i / dk, d = i % dk;
            K[j * ldk + d] = k0 + j < k_end ? to_f(((const T*)a.k)[(long long)(krow + k0 + j) * a.ldk + hk * dk + d]) : 0.f;
        }
        for (int i = threadIdx.x; i < TK * dv; i += NT) {
            const int j = i / dv, d = i % dv;
            V[i] = k0 + j < k_end ? to_f(((const T*)a.v)[(long long)(krow + k0 + j) * a.ldv + hv * dv + d]) : 0.f;
        }
        __syncthreads();
        float s[KP];
#pragma unroll
        for (int e = 0; e < KP; ++e) s[e] = 0.f;
        for (int d = 0; d < dk; ++d) {
            const float q = Q[r * ldk + d];
#pragma unroll
            for (int e = 0; e < KP; ++e) s[e] += q * K[(part + 4 * e) * ldk + d];
        }
        float mx = m, corr = 1.f;
        if (a.bias != nullptr) {
#pragma unroll
            for (int e = 0; e < KP; ++e) {
                const int key = k0 + part + 4 * e;
                const bool seen = key <= qi && (a.window <= 0 || key > qi - a.window);
                S[r * (TK + 1) + part + 4 * e] = seen ? a.mul / (1.f + expf(-(s[e] * a.scale + a.bias[h]))) : 0.f;
            }
            l = 1.f;
        } else {
#pragma unroll
            for (int e = 0; e < KP; ++e) {
                const int key = k0 + part + 4 * e;
                s[e] = key <= qi && (a.window <= 0 || key > qi - a.window) ? s[e] * a.scale : -INFINITY;
                mx = fmaxf(mx, s[e]);
            }
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
            corr = m == -INFINITY ? 0.f : expf(m - mx);
            float ps = 0.f;
#pragma unroll
            for (int e = 0; e < KP; ++e) {
                const float p = mx == -INFINITY ? 0.f : expf(s[e] - mx);   // no visible key yet
                S[r * (TK + 1) + part + 4 * e] = p;
                ps += p;
            }
            ps += __shfl_xor_sync(0xffffffffu, ps, 1);
            ps += __shfl_xor_sync(0xffffffffu, ps, 2);
            l = l * corr + ps;
            m = mx;
        }
        __syncwarp();
        for (int d = part; d < dv; d += 4) {
            float o = O[r * dv + d] * corr;
            for (int j = 0; j < TK; ++j) o += S[r * (TK + 1) + j] * V[j * dv + d];
            O[r * dv + d] = o;
        }
        __syncwarp();
    }
    if (r < nq) {
        T* out = (T*)a.out + (row0 + r) * a.ldo + ho * dv;
        const T* g = a.gate == nullptr ? nullptr : (const T*)a.gate + (row0 + r) * a.ldg + h * dv;
        for (int d = part; d < dv; d += 4) {
            const float o = O[r * dv + d] / l;
            out[d] = from_f<T>(g == nullptr ? o : o / (1.f + expf(-to_f(g[d]))));
        }
    }
}

template <typename T, int TQ>
static int launch_rows(const Prompt& a, cudaStream_t st) {
    const size_t smem = sizeof(float) * (2 * TQ * (size_t)(a.dk + 1) + 2 * TQ * (size_t)a.dv + TQ * (TQ + 1));
    if (smem > 227 * 1024) return -2;
    cudaError_t e = cudaFuncSetAttribute(packed_attn_rows_kernel<T, TQ>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    packed_attn_rows_kernel<T, TQ><<<dim3(a.n, a.H, a.cross ? a.G : 1), TQ * 4, smem, st>>>(a);
    return (int)cudaGetLastError();
}

// ---------------------------------------------------------------------------------------------------------------- one token
constexpr int ST = 256, SK = 64;         // threads, keys per tile

// grid (H, n, cross ? G : 1)
template <typename T>
__global__ void __launch_bounds__(ST) packed_attn_step_kernel(Step a) {
    extern __shared__ float sm[];
    float* Q = sm;                       // [dk]
    float* O = Q + a.dk;                 // [dv]
    float* P = O + a.dv;                 // [SK]
    __shared__ long long rows[SK];
    __shared__ float red[32];
    const int h = blockIdx.x, b = blockIdx.y, hk = h / (a.H / a.G);
    const int hv = a.cross ? blockIdx.z : hk, ho = a.cross ? h * a.G + hv : h;
    const int w = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int slot = a.slots[b], pos = a.pos[b];
    const int first = a.c.table == nullptr ? max(0, pos + 1 - a.c.cap) : a.window > 0 ? max(0, pos + 1 - a.window) : 0;
    const T* q = (const T*)a.q + (long long)b * a.ldq + (long long)h * a.dk;
    for (int d = threadIdx.x; d < a.dk; d += ST) Q[d] = to_f(q[d]);
    for (int d = threadIdx.x; d < a.dv; d += ST) O[d] = 0.f;
    float m = -INFINITY, l = 0.f;
    for (int k0 = first; k0 <= pos; k0 += SK) {
        const int nt = min(SK, pos + 1 - k0);
        __syncthreads();
        if (threadIdx.x < nt) rows[threadIdx.x] = a.c.row(slot, k0 + threadIdx.x) * a.G;
        __syncthreads();
        for (int j = w; j < nt; j += ST / 32) {
            const T* k = (const T*)a.c.k + (rows[j] + hk) * a.dk;
            float s = 0.f;
            for (int d = lane; d < a.dk; d += 32) s += Q[d] * to_f(k[d]);
            s = warp_sum(s);
            if (lane == 0) P[j] = s * a.scale;
        }
        __syncthreads();
        float corr = 1.f;
        if (a.bias != nullptr) {
            if (threadIdx.x < nt) P[threadIdx.x] = a.mul / (1.f + expf(-(P[threadIdx.x] + a.bias[h])));
            l = 1.f;
            __syncthreads();
        } else {
            const float x = threadIdx.x < nt ? P[threadIdx.x] : -INFINITY;
            const float mx = fmaxf(m, block_max(x, red));
            const float p = threadIdx.x < nt ? expf(x - mx) : 0.f;
            if (threadIdx.x < nt) P[threadIdx.x] = p;
            const float ps = block_sum(p, red);              // also orders the writes of P
            corr = m == -INFINITY ? 0.f : expf(m - mx);
            l = l * corr + ps;
            m = mx;
        }
        for (int d = threadIdx.x; d < a.dv; d += ST) {
            float o = O[d] * corr;
            for (int j = 0; j < nt; ++j) o += P[j] * to_f(((const T*)a.c.v)[(rows[j] + hv) * a.dv + d]);
            O[d] = o;
        }
    }
    T* out = (T*)a.out + (long long)b * a.ldo + (long long)ho * a.dv;
    for (int d = threadIdx.x; d < a.dv; d += ST) out[d] = from_f<T>(O[d] / l);
}

template <typename T>
static int launch_step(const Step& a, cudaStream_t st) {
    const size_t smem = sizeof(float) * (a.dk + a.dv + SK);
    if (smem > 200 * 1024) return -2;
    cudaError_t e = cudaFuncSetAttribute(packed_attn_step_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    packed_attn_step_kernel<T><<<dim3(a.H, a.n, a.cross ? a.G : 1), ST, smem, st>>>(a);
    return (int)cudaGetLastError();
}

// --------------------------------------------------------------------------------------------------------------- row kernels
constexpr int THREADS = 256;

struct QkNorm {
    void* z;                             // [rows, ldz]: queries (H x dk), keys (G x dk), values (G x dv) from columns zq, zk, zv
    const float *wq, *wk;                // norm weights [H * dk], [G * dk] (null: no norm)
    const double* freq;                  // [rot / 2] rotation per position (null: no rotation)
    Cache c;                             // k null: nothing is stored
    const int *pos, *slots, *ends;       // [rows]; ends: length of the request after this call, null: store every row
    long long ldz;
    int zq, zk, zv, H, G, dk, dv;        // dk, dv as laid out (padded with zero columns)
    int nq, nk;                          // numbers in a norm (H, G x the unpadded size)
    int rot;
    float eps;
    int rows;
};

// sums of two numbers per thread over the block; red: 16 float2
__device__ __forceinline__ float2 block_sum2(float2 v, float2* red) {
    v.x = warp_sum(v.x);
    v.y = warp_sum(v.y);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    v = make_float2(0.f, 0.f);
    for (int i = 0; i < THREADS / 32; ++i) {
        v.x += red[i].x;
        v.y += red[i].y;
    }
    return v;
}

template <typename T>
__global__ void __launch_bounds__(THREADS) qk_norm_rope_kernel(QkNorm a) {
    pdl_trigger();
    constexpr int W = Vec<T>::N, NV = sizeof(T) == 2 ? 3 : 2;           // pieces a thread keeps in registers
    extern __shared__ float2 turn[];     // [rot / 2] (cos, sin)
    __shared__ float2 red[THREADS / 32];
    const int row = blockIdx.x, pos = a.pos[row];
    const int nq = a.H * a.dk, n = nq + a.G * a.dk;                     // queries, then keys
    T* z = (T*)a.z + (long long)row * a.ldz;
    auto at = [&](int i) { return z + (i < nq ? a.zq + i : a.zk + i - nq); };
    Vec<T> v[NV];
#pragma unroll
    for (int t = 0; t < NV; ++t) {
        const int i = (threadIdx.x + t * THREADS) * W;
        if (i < n) v[t].load(at(i));
    }
    for (int i = threadIdx.x; i < a.rot / 2; i += THREADS) {
        // range reduction in double: the angle is exact to fp32 at any position
        constexpr double TWO_PI = 6.283185307179586476925286766559, INV = 0.15915494309189533576888376337251;
        const double angle = (double)pos * a.freq[i];
        const float r = (float)(angle - TWO_PI * rint(angle * INV));
        turn[i] = make_float2(cosf(r), sinf(r));
    }
    float2 sum = make_float2(0.f, 0.f);
    auto square = [&](const Vec<T>& x, int i) {
        float s = 0.f;
#pragma unroll
        for (int e = 0; e < W; ++e) s += x.get(e) * x.get(e);
        if (i < nq) sum.x += s;
        else sum.y += s;
    };
#pragma unroll
    for (int t = 0; t < NV; ++t) {
        const int i = (threadIdx.x + t * THREADS) * W;
        if (i < n) square(v[t], i);
    }
    for (int i = (threadIdx.x + NV * THREADS) * W; i < n; i += THREADS * W) {
        Vec<T> x;
        x.load(at(i));
        square(x, i);
    }
    sum = block_sum2(sum, red);                                         // its barrier also covers `turn`
    const float rq = 1.f / sqrtf(sum.x / a.nq + a.eps), rk = 1.f / sqrtf(sum.y / a.nk + a.eps);
    T* kd = nullptr;
    T* vd = nullptr;
    // a ring keeps the request's last `cap` positions: of the rows that share a place only the last one is stored
    if (a.c.k != nullptr && (a.ends == nullptr || a.c.table != nullptr || pos >= a.ends[row] - a.c.cap)) {
        const long long r = a.c.row(a.slots[row], pos) * a.G;
        kd = (T*)a.c.k + r * a.dk;
        vd = (T*)a.c.v + r * a.dv;
    }
    auto finish = [&](Vec<T>& x, int i) {
        const bool is_q = i < nq;
        const int c = is_q ? i : i - nq, d = c % a.dk;
        const float* weight = is_q ? a.wq : a.wk;
        const float r = is_q ? rq : rk;
        float f[W];
#pragma unroll
        for (int e = 0; e < W; ++e) f[e] = weight == nullptr ? x.get(e) : x.get(e) * r * weight[c + e];
#pragma unroll
        for (int e = 0; e < W; e += 2) {
            if (d + e < a.rot) {
                const float2 cs = turn[(d + e) / 2];
                const float u = f[e], t = f[e + 1];
                f[e] = u * cs.x - t * cs.y;
                f[e + 1] = t * cs.x + u * cs.y;
            }
        }
#pragma unroll
        for (int e = 0; e < W; ++e) x.set(e, f[e]);
        x.store(at(i));
        if (!is_q && kd != nullptr) x.store(kd + c);
    };
#pragma unroll
    for (int t = 0; t < NV; ++t) {
        const int i = (threadIdx.x + t * THREADS) * W;
        if (i < n) finish(v[t], i);
    }
    for (int i = (threadIdx.x + NV * THREADS) * W; i < n; i += THREADS * W) {
        Vec<T> x;
        x.load(at(i));
        finish(x, i);
    }
    if (vd != nullptr)
        for (int i = threadIdx.x * W; i < a.G * a.dv; i += THREADS * W) {
            Vec<T> x;
            x.load(z + a.zv + i);
            x.store(vd + i);
        }
}

struct HeadNorm {
    void* z;                             // [rows, ldz]: queries (H x dk), keys (G x dk), values (V x dv) from columns zq, zk, zv
    const float *wq, *wk;                // norm weights [dk], shared by the heads (null: no norm)
    const float2* turn;                  // [rows, rot / 2] (cos, sin)
    const void* first;                   // [rows, ldf]: v <- (1 - *mix) v + *mix first (null: values as they are)
    const float* mix;
    Cache c;                             // k null: nothing is stored
    const int *pos, *slots, *ends;       // as in QkNorm
    long long ldz, ldf;
    int zq, zk, zv, H, G, V, dk, dv;     // V: G, or 0: no values
    int nk, nv;                          // numbers in a norm (the unpadded head sizes)
    int rot, halves;                     // rotated dimensions; pairs (i, i + rot / 2) or neighbours
    int norm_v;
    float eps;
    int rows;
};

// turn [rows, half] = size (cos, sin) of pos * freq
__global__ void __launch_bounds__(THREADS) rotary_rows_kernel(const int* __restrict__ pos, const double* __restrict__ freq, float2* __restrict__ turn, int rows,
                                                              int half, float size) {
    pdl_trigger();
    for (long long i = blockIdx.x * (long long)THREADS + threadIdx.x; i < (long long)rows * half; i += (long long)gridDim.x * THREADS) {
        // range reduction in double: the angle is exact to fp32 at any position
        constexpr double TWO_PI = 6.283185307179586476925286766559, INV = 0.15915494309189533576888376337251;
        const double angle = (double)pos[i / half] * freq[i % half];
        const float r = (float)(angle - TWO_PI * rint(angle * INV));
        turn[i] = make_float2(cosf(r) * size, sinf(r) * size);
    }
}

// grid (rows, parts): a warp takes every (8 parts)-th head; the head lies in shared memory in fp32 between the norm and the rotation
template <typename T>
__global__ void __launch_bounds__(THREADS) head_norm_rope_kernel(HeadNorm a) {
    pdl_trigger();
    extern __shared__ float4 sm4[];      // one head per warp
    const int row = blockIdx.x, pos = a.pos[row], w = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int half = a.rot / 2, heads = a.H + a.G + a.V, size = max(a.dk, a.dv), stride = gridDim.y * (THREADS / 32);
    float* X = reinterpret_cast<float*>(sm4) + w * size;
    const float2* turn = a.turn + (long long)row * half;
    T* z = (T*)a.z + (long long)row * a.ldz;
    auto start = [&](int i) { return z + (i < a.H ? a.zq + i * a.dk : i < a.H + a.G ? a.zk + (i - a.H) * a.dk : a.zv + (i - a.H - a.G) * a.dv); };
    int i = blockIdx.y * (THREADS / 32) + w;
    float4 ahead = make_float4(0.f, 0.f, 0.f, 0.f);          // the first piece of this warp's next head
    if (i < heads && lane * 4 < (i < a.H + a.G ? a.dk : a.dv)) ahead = load4(start(i) + lane * 4);
    // a ring keeps the request's last `cap` positions: of the rows that share a place only the last one is stored
    const bool store = a.c.k != nullptr && (a.ends == nullptr || a.c.table != nullptr || pos >= a.ends[row] - a.c.cap);
    const long long place = store ? a.c.row(a.slots[row], pos) * a.G : 0;
    const float mix = a.first != nullptr ? *a.mix : 0.f;
    const bool aligned = a.halves && half % 4 == 0;          // four neighbours lie in one half, and so do their partners
    for (; i < heads; i += stride) {
        const bool is_v = i >= a.H + a.G, is_k = !is_v && i >= a.H;
        const int n = is_v ? a.dv : a.dk;
        T* p = start(i);
        float s = 0.f;
        for (int c = lane * 4; c < n; c += 128) {
            const float4 x = c == lane * 4 ? ahead : load4(p + c);
            s += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
            *reinterpret_cast<float4*>(X + c) = x;
        }
        if (i + stride < heads && lane * 4 < (i + stride < a.H + a.G ? a.dk : a.dv)) ahead = load4(start(i + stride) + lane * 4);
        s = warp_sum(s);
        __syncwarp();
        const float* weight = is_v ? nullptr : is_k ? a.wk : a.wq;
        const float r = (is_v ? a.norm_v != 0 : weight != nullptr) ? 1.f / sqrtf(s / (is_v ? a.nv : a.nk) + a.eps) : 1.f;
        auto number = [&](int d) { return X[d] * r * (weight == nullptr ? 1.f : weight[d]); };
        auto four = [&](int d) {
            const float4 x = *reinterpret_cast<const float4*>(X + d), g = weight == nullptr ? make_float4(1.f, 1.f, 1.f, 1.f) : load4(weight + d);
            return make_float4(x.x * r * g.x, x.y * r * g.y, x.z * r * g.z, x.w * r * g.w);
        };
        T* cached = !store || i < a.H ? nullptr : is_v ? (T*)a.c.v + (place + i - a.H - a.G) * a.dv : (T*)a.c.k + (place + i - a.H) * a.dk;
        const T* other = is_v && a.first != nullptr ? (const T*)a.first + (long long)row * a.ldf + (i - a.H - a.G) * a.dv : nullptr;
        for (int c = lane * 4; c < n; c += 128) {
            float4 y = four(c);
            if (!is_v && c < a.rot) {
                if (aligned) {
                    const bool low = c < half;
                    const float4 o = four(low ? c + half : c - half);
                    const float4* t = reinterpret_cast<const float4*>(turn + (low ? c : c - half));
                    const float4 t0 = t[0], t1 = t[1];       // (cos, sin) of four pairs
                    const float sign = low ? -1.f : 1.f;
                    y = make_float4(y.x * t0.x + sign * o.x * t0.y, y.y * t0.z + sign * o.y * t0.w, y.z * t1.x + sign * o.z * t1.y,
                                    y.w * t1.z + sign * o.w * t1.w);
                } else {
                    float f[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int d = c + e;
                        if (d < a.rot) {
                            const bool low = a.halves ? d < half : (d & 1) == 0;
                            const float2 t = turn[a.halves ? (low ? d : d - half) : d >> 1];
                            const float o = number(a.halves ? (low ? d + half : d - half) : d ^ 1);
                            f[e] = low ? f[e] * t.x - o * t.y : f[e] * t.x + o * t.y;
                        }
                    }
                    y = make_float4(f[0], f[1], f[2], f[3]);
                }
            }
            if (other != nullptr) {
                const float4 o = load4(other + c);
                y = make_float4((1.f - mix) * y.x + mix * o.x, (1.f - mix) * y.y + mix * o.y, (1.f - mix) * y.z + mix * o.z, (1.f - mix) * y.w + mix * o.w);
            }
            store4(p + c, y);
            if (cached != nullptr) store4(cached + c, y);
        }
        __syncwarp();
    }
}

// x [n, ldx]: [H, G, dv] per row -> out [n, ldo]: out[h] = sum over g of table[h, g] x[g, value head of h].  A thread takes 16 bytes of a
// value head and HT of the heads that share it (HT divides their number).
template <typename T, int HT>
__global__ void __launch_bounds__(THREADS) head_mix_kernel(const T* __restrict__ x, long long ldx, const float* __restrict__ table, T* __restrict__ out,
                                                           long long ldo, int n, int H, int G, int dv) {
    pdl_trigger();
    constexpr int W = Vec<T>::N, AHEAD = 8;                  // softmax heads whose pieces are in flight
    extern __shared__ float sm[];                            // [H][H] transposed: [g][h]
    for (int i = threadIdx.x; i < H * H; i += THREADS) sm[i % H * H + i / H] = table[i];
    __syncthreads();
    const int qpg = H / G, pieces = dv / W, tiles = qpg / HT, per_row = G * tiles * pieces;
    const long long total = (long long)n * per_row, pitch = (long long)G * dv;
    for (long long i = blockIdx.x * (long long)THREADS + threadIdx.x; i < total; i += (long long)gridDim.x * THREADS) {
        const long long row = i / per_row;
        const int in_row = (int)(i - row * per_row), c = in_row % pieces * W, k = in_row / pieces % G, h0 = k * qpg + in_row / pieces / G * HT;
        float acc[HT][W];
#pragma unroll
        for (int h = 0; h < HT; ++h)
#pragma unroll
            for (int e = 0; e < W; ++e) acc[h][e] = 0.f;
        const T* p = x + row * ldx + k * dv + c;
        for (int g0 = 0; g0 < H; g0 += AHEAD) {
            Vec<T> v[AHEAD];
#pragma unroll
            for (int j = 0; j < AHEAD; ++j) v[j].load(p + min(g0 + j, H - 1) * pitch);
#pragma unroll
            for (int j = 0; j < AHEAD; ++j) {
                if (g0 + j < H) {
                    const float* t = sm + (g0 + j) * H + h0;
                    float f[W];
#pragma unroll
                    for (int e = 0; e < W; ++e) f[e] = v[j].get(e);
#pragma unroll
                    for (int h = 0; h < HT; ++h) {
                        const float w = t[h];
#pragma unroll
                        for (int e = 0; e < W; ++e) acc[h][e] += w * f[e];
                    }
                }
            }
        }
#pragma unroll
        for (int h = 0; h < HT; ++h) {
            Vec<T> y;
#pragma unroll
            for (int e = 0; e < W; ++e) y.set(e, acc[h][e]);
            y.store(out + row * ldo + (long long)(h0 + h) * dv + c);
        }
    }
}

template <typename T, int HT>
static int launch_mix(const void* x, long long ldx, const float* table, void* out, long long ldo, int n, int H, int G, int dv, cudaStream_t st) {
    const size_t smem = sizeof(float) * H * H;
    if (smem > 227 * 1024) return -2;
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(head_mix_kernel<T, HT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    const long long total = (long long)n * (H / HT) * (dv / Vec<T>::N), blocks = (total + THREADS - 1) / THREADS;
    head_mix_kernel<T, HT><<<(unsigned)(blocks < 148 * 16 ? blocks : 148 * 16), THREADS, smem, st>>>((const T*)x, ldx, table, (T*)out, ldo, n, H, G, dv);
    return (int)cudaGetLastError();
}

template <typename T>
static int mix_by_heads(const void* x, long long ldx, const float* table, void* out, long long ldo, int n, int H, int G, int dv, cudaStream_t st) {
    const int qpg = H / G;
    return qpg % 4 == 0   ? launch_mix<T, 4>(x, ldx, table, out, ldo, n, H, G, dv, st)
           : qpg % 3 == 0 ? launch_mix<T, 3>(x, ldx, table, out, ldo, n, H, G, dv, st)
           : qpg % 2 == 0 ? launch_mix<T, 2>(x, ldx, table, out, ldo, n, H, G, dv, st)
                          : launch_mix<T, 1>(x, ldx, table, out, ldo, n, H, G, dv, st);
}

struct LatentNorm {
    const void* z;                       // [rows, ldz], latent projection from column 0 (pitch ldz)
    void* c;                             // [rows, ldc] normed rows
    const float* weight;                 // [rank]
    Cache cache;                         // k null: nothing is stored
    const int *pos, *slots;
    long long ldz, ldc;
    int width, rank;                     // columns as laid out (padded with zeros), numbers in the norm
    float eps;
    int rows;
};

// one warp per row
template <typename T>
__global__ void __launch_bounds__(128) latent_norm_kernel(LatentNorm a) {
    pdl_trigger();
    constexpr int W = Vec<T>::N, NV = 16 / W * 2;            // pieces a lane keeps in registers (rows up to 1024 wide)
    const int row = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (row >= a.rows) return;
    const T* z = (const T*)a.z + (long long)row * a.ldz;
    T* c = (T*)a.c + (long long)row * a.ldc;
    T* dst = a.cache.k == nullptr ? nullptr : (T*)a.cache.k + a.cache.row(a.slots[row], a.pos[row]) * a.width;
    Vec<T> v[NV];
    float s = 0.f;
    auto square = [&](const Vec<T>& x) {
#pragma unroll
        for (int e = 0; e < W; ++e) s += x.get(e) * x.get(e);
    };
#pragma unroll
    for (int t = 0; t < NV; ++t) {
        const int i = (lane + t * 32) * W;
        if (i < a.width) v[t].load(z + i);
    }
#pragma unroll
    for (int t = 0; t < NV; ++t)
        if ((lane + t * 32) * W < a.width) square(v[t]);
    for (int i = (lane + NV * 32) * W; i < a.width; i += 32 * W) {
        Vec<T> x;
        x.load(z + i);
        square(x);
    }
    const float r = 1.f / sqrtf(warp_sum(s) / a.rank + a.eps);
    auto finish = [&](Vec<T>& x, int i) {
#pragma unroll
        for (int e = 0; e < W; ++e) x.set(e, x.get(e) * r * a.weight[i + e]);
        x.store(c + i);
        if (dst != nullptr) x.store(dst + i);
    };
#pragma unroll
    for (int t = 0; t < NV; ++t) {
        const int i = (lane + t * 32) * W;
        if (i < a.width) finish(v[t], i);
    }
    for (int i = (lane + NV * 32) * W; i < a.width; i += 32 * W) {
        Vec<T> x;
        x.load(z + i);
        finish(x, i);
    }
}

// meta [n, 4]: {destination row, source row of `src` or -1, slot, position}
template <typename T>
__global__ void __launch_bounds__(128) gather_rows_kernel(T* dst, long long ldd, const T* src, long long lds, Cache c, int cols,
                                                          const int4* __restrict__ meta) {
    constexpr int W = Vec<T>::N;
    const int4 e = meta[blockIdx.x];
    const T* s = e.y >= 0 ? src + e.y * lds : (const T*)c.k + c.row(e.z, e.w) * cols;
    T* d = dst + e.x * ldd;
    for (int i = threadIdx.x * W; i < cols; i += 128 * W) {
        Vec<T> v;
        v.load(s + i);
        v.store(d + i);
    }
}

template <typename T>
__global__ void __launch_bounds__(THREADS) gate_rows_kernel(T* o, long long ldo, const T* g, long long ldg, int cols) {
    T* orow = o + (long long)blockIdx.x * ldo;
    const T* grow = g + (long long)blockIdx.x * ldg;
    for (int i = threadIdx.x; i < cols; i += THREADS) orow[i] = from_f<T>(to_f(orow[i]) / (1.f + expf(-to_f(grow[i]))));
}

static bool aligned(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

}  // namespace pag
}  // namespace lmoe

using namespace lmoe;

// dt: 1 bf16, 0 fp32.  Work items of `tile` (32 or 16) queries at most; scale of any sign.
LMOE_API int lmoe_packed_attn_rows(const pa::Prompt* ap, int tile, int dt, cudaStream_t st) {
    const pa::Prompt& a = *ap;
    if (a.n <= 0 || a.H <= 0 || a.G <= 0 || a.H % a.G || a.dk <= 0 || a.dv <= 0) return -1;
    if (tile == 32) return dt ? pag::launch_rows<bf16, 32>(a, st) : pag::launch_rows<float, 32>(a, st);
    if (tile == 16) return dt ? pag::launch_rows<bf16, 16>(a, st) : pag::launch_rows<float, 16>(a, st);
    return -1;
}

LMOE_API int lmoe_packed_attn_step_any(const pa::Step* ap, int dt, cudaStream_t st) {
    const pa::Step& a = *ap;
    if (a.n <= 0 || a.H <= 0 || a.G <= 0 || a.H % a.G || a.dk <= 0 || a.dv <= 0 || (a.c.table == nullptr && a.c.cap <= 0)) return -1;
    return dt ? pag::launch_step<bf16>(a, st) : pag::launch_step<float>(a, st);
}

// dk, dv, ldz and the first columns multiples of 8 (bf16) or 4 (fp32), rot even
LMOE_API int lmoe_qk_norm_rope(const pag::QkNorm* ap, int dt, cudaStream_t st) {
    const pag::QkNorm& a = *ap;
    const int w = dt ? 8 : 4;
    if (a.rows <= 0 || a.H <= 0 || a.G <= 0 || a.dk % w || a.dv % w || a.ldz % w || a.zq % w || a.zk % w || a.zv % w || a.rot % 2 || a.rot < 0 ||
        a.rot > a.dk || a.nq <= 0 || a.nk <= 0 || !pag::aligned(a.z) || !pag::aligned(a.c.k) || !pag::aligned(a.c.v) ||
        (a.c.k != nullptr && a.c.table == nullptr && a.c.cap <= 0) || (a.rot > 0 && a.freq == nullptr))
        return -1;
    const size_t smem = sizeof(float2) * (a.rot / 2);
    if (smem > 40 * 1024) return -2;
    if (dt) pag::qk_norm_rope_kernel<bf16><<<a.rows, pag::THREADS, smem, st>>>(a);
    else pag::qk_norm_rope_kernel<float><<<a.rows, pag::THREADS, smem, st>>>(a);
    return (int)cudaGetLastError();
}

// pos [rows], freq [half] -> turn [rows, half] (cos, sin) times size
LMOE_API int lmoe_rotary_rows(const int* pos, const double* freq, void* turn, int rows, int half, float size, cudaStream_t st) {
    if (rows <= 0 || half <= 0 || !pag::aligned(turn)) return -1;
    const long long blocks = ((long long)rows * half + pag::THREADS - 1) / pag::THREADS;
    pag::rotary_rows_kernel<<<(unsigned)(blocks < 148 * 32 ? blocks : 148 * 32), pag::THREADS, 0, st>>>(pos, freq, (float2*)turn, rows, half, size);
    return (int)cudaGetLastError();
}

// dk, dv, ldz, ldf and the first columns multiples of 8 (bf16) or 4 (fp32), rot even
LMOE_API int lmoe_head_norm_rope(const pag::HeadNorm* ap, int dt, cudaStream_t st) {
    const pag::HeadNorm& a = *ap;
    const int w = dt ? 8 : 4;
    if (a.rows <= 0 || a.H <= 0 || a.G <= 0 || (a.V != 0 && a.V != a.G) || a.dk <= 0 || a.dk % w || a.dv < 0 || a.dv % w || a.ldz % w || a.ldf % w || a.zq % w ||
        a.zk % w || a.zv % w || a.rot % 2 || a.rot < 0 || a.rot > a.dk || a.nk <= 0 || (a.V && a.nv <= 0) || !pag::aligned(a.z) || !pag::aligned(a.first) ||
        !pag::aligned(a.wq) || !pag::aligned(a.wk) || !pag::aligned(a.c.k) || !pag::aligned(a.c.v) ||
        (a.c.k != nullptr && ((a.c.table == nullptr && a.c.cap <= 0) || !a.V)) || (a.rot > 0 && a.turn == nullptr) || !pag::aligned(a.turn) || (a.first != nullptr && a.mix == nullptr))
        return -1;
    const size_t smem = sizeof(float) * (pag::THREADS / 32) * (a.dk > a.dv ? a.dk : a.dv);
    if (smem > 46 * 1024) return -2;
    const int heads = a.H + a.G + a.V, parts = a.rows >= 1024 ? 1 : (heads + 7) / 8;
    if (dt) pag::head_norm_rope_kernel<bf16><<<dim3(a.rows, parts), pag::THREADS, smem, st>>>(a);
    else pag::head_norm_rope_kernel<float><<<dim3(a.rows, parts), pag::THREADS, smem, st>>>(a);
    return (int)cudaGetLastError();
}

// x [n, ldx] with H * G * dv columns -> out [n, ldo] with H * dv columns; table [H, H]; dv and pitches multiples of 8 (bf16) or 4 (fp32)
LMOE_API int lmoe_head_mix(const void* x, long long ldx, const float* table, void* out, long long ldo, int n, int H, int G, int dv, int dt,
                           cudaStream_t st) {
    const int w = dt ? 8 : 4;
    if (n <= 0 || H <= 0 || G <= 0 || H % G || dv <= 0 || dv % w || ldx % w || ldo % w || !pag::aligned(x) || !pag::aligned(out)) return -1;
    return dt ? pag::mix_by_heads<bf16>(x, ldx, table, out, ldo, n, H, G, dv, st) : pag::mix_by_heads<float>(x, ldx, table, out, ldo, n, H, G, dv, st);
}

LMOE_API int lmoe_latent_norm(const pag::LatentNorm* ap, int dt, cudaStream_t st) {
    const pag::LatentNorm& a = *ap;
    const int w = dt ? 8 : 4;
    if (a.rows <= 0 || a.width <= 0 || a.rank <= 0 || a.width % w || a.ldz % w || a.ldc % w || !pag::aligned(a.z) || !pag::aligned(a.c) ||
        !pag::aligned(a.cache.k) || (a.cache.k != nullptr && a.cache.table == nullptr && a.cache.cap <= 0))
        return -1;
    if (dt) pag::latent_norm_kernel<bf16><<<(a.rows + 3) / 4, 128, 0, st>>>(a);
    else pag::latent_norm_kernel<float><<<(a.rows + 3) / 4, 128, 0, st>>>(a);
    return (int)cudaGetLastError();
}

// cols: row length in both places; the cache rows are the request's whole rows (all kv heads)
LMOE_API int lmoe_gather_rows(void* dst, long long ldd, const void* src, long long lds, const pa::Cache* c, int cols, const int* meta, int n,
                              int dt, cudaStream_t st) {
    const int w = dt ? 8 : 4;
    if (n <= 0 || cols <= 0 || cols % w || ldd % w || lds % w || !pag::aligned(dst) || !pag::aligned(src) || !pag::aligned(meta)) return -1;
    if (dt) pag::gather_rows_kernel<bf16><<<n, 128, 0, st>>>((bf16*)dst, ldd, (const bf16*)src, lds, *c, cols, (const int4*)meta);
    else pag::gather_rows_kernel<float><<<n, 128, 0, st>>>((float*)dst, ldd, (const float*)src, lds, *c, cols, (const int4*)meta);
    return (int)cudaGetLastError();
}

LMOE_API int lmoe_gate_rows(void* o, long long ldo, const void* g, long long ldg, int rows, int cols, int dt, cudaStream_t st) {
    if (rows <= 0 || cols <= 0) return -1;
    if (dt) pag::gate_rows_kernel<bf16><<<rows, pag::THREADS, 0, st>>>((bf16*)o, ldo, (const bf16*)g, ldg, cols);
    else pag::gate_rows_kernel<float><<<rows, pag::THREADS, 0, st>>>((float*)o, ldo, (const float*)g, ldg, cols);
    return (int)cudaGetLastError();
}
