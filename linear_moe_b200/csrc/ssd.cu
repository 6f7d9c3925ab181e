// State-space duality (Mamba-2) over packed rows: a short convolution, S <- exp(-exp(A) dt) S + dt B x^T with y = S^T C + D x head by head in
// fp32, then a gated norm:
//   ssd_conv_kernel   prompts: x, B and C behind the convolution and SiLU; step sizes and log decays
//   ssd_tail_kernel   prompts: the last inputs of the convolution -> the cache
//   ssd_scan_kernel   prompts of any size, bf16 or fp32, token by token (bf16 fast path: ssd_tc.cu)
//   ssd_step_kernel   one token per request: convolution, step size and state update in one pass over the state
//   ssd_norm_kernel   y silu(z) over the root mean square of its part of the row, times weight and factor
// Compiled without fast-math: the fp32 instantiations serve models in true 32-bit.
#include "mma_utils.cuh"
#include "ssd.cuh"

namespace lmoe {
namespace ssd {

// as exactly as the model's type asks for
template <typename T> __device__ __forceinline__ float silu(float x) { return sizeof(T) == 2 ? __fdividef(x, 1.f + __expf(-x)) : x / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// ------------------------------------------------------------------------------------------------------- prompts: convolution
constexpr int CT = 128, CROWS = 16;      // threads, rows of a CTA

// grid (row tiles, pieces of 4 channels per thread).  A thread slides over CROWS rows of its channels with the last inputs in registers.
template <typename T, int TAPS>
__global__ void __launch_bounds__(CT) ssd_conv_kernel(Args a) {
    pdl_trigger();
    constexpr int W = 4;
    const int ch = a.channels(), c = (blockIdx.y * CT + threadIdx.x) * W;
    const int r0 = blockIdx.x * CROWS, r1 = min(a.rows, r0 + CROWS);
    if (blockIdx.y == 0) {                                   // step sizes
        for (int i = threadIdx.x; i < (r1 - r0) * a.H; i += CT) {
            const int row = r0 + i / a.H, h = i % a.H;
            const float dt = softplus(to_f(((const T*)a.z)[row * a.ldz + a.zdt + h]) + a.dt_bias[h]);
            a.dt[(long long)row * a.H + h] = dt;
            a.la[(long long)row * a.H + h] = -expf(a.a_log[h]) * dt;
        }
    }
    if (c >= ch) return;
    const int taps = TAPS ? TAPS : a.taps;
    constexpr int KEEP = TAPS ? TAPS : MAX_TAPS;
    const T* z = (const T*)a.z + a.zx + c;
    float4 w[KEEP], past[KEEP];                              // past[n]: the input n + 1 positions back
#pragma unroll
    for (int n = 0; n < KEEP; ++n)
        if (n < taps) w[n] = load4(a.conv + (long long)n * ch + c);
    const float4 bias = load4(a.conv_bias + c), zero = make_float4(0.f, 0.f, 0.f, 0.f);
    auto input = [&](int row, int back) {                    // of the same request, `back` positions in front of row
        const int p = a.pos[row] - back;
        if (p < 0) return zero;
        // rows of a request are consecutive and its positions count up: the row `back` earlier is its own if the positions say so
        const int e = row - back;
        if (e >= 0 && a.pos[e] == p && a.slots[e] == a.slots[row]) return load4(z + e * a.ldz);
        return a.tail == nullptr ? zero : load4((const T*)a.tail + ((long long)a.slots[row] * a.ring + p % a.ring) * ch + c);
    };
    int last = -2;                                           // position of the previous row
    for (int row = r0; row < r1; ++row) {
        const int pos = a.pos[row];
        if (row == r0 || pos != last + 1 || a.slots[row] != a.slots[row - 1]) {
#pragma unroll
            for (int n = 0; n < KEEP; ++n)
                if (n + 1 < taps) past[n] = input(row, n + 1);
        }
        last = pos;
        const float4 x = load4(z + row * a.ldz);
        float4 s = bias;
#pragma unroll
        for (int n = 0; n < KEEP; ++n)
            if (n < taps) {
                const float4 v = n == 0 ? x : past[n > 0 ? n - 1 : 0];
                // tap taps - 1 - n meets the input n positions back
                const float4 k = TAPS ? w[(TAPS ? TAPS : 1) - 1 - n] : load4(a.conv + (long long)(taps - 1 - n) * ch + c);
                s.x += k.x * v.x; s.y += k.y * v.y; s.z += k.z * v.z; s.w += k.w * v.w;
            }
#pragma unroll
        for (int n = KEEP - 1; n > 0; --n) past[n] = past[n - 1];
        past[0] = x;
        store4((T*)a.xbc + row * a.ldx + c, make_float4(silu<T>(s.x), silu<T>(s.y), silu<T>(s.z), silu<T>(s.w)));
    }
}

// grid (requests, taps): the input blockIdx.y rows in front of a request's last new one
template <typename T>
__global__ void __launch_bounds__(CT) ssd_tail_kernel(Args a) {
    pdl_trigger();
    const int ch = a.channels();
    int row, n = 1, slot;
    if (a.groups != nullptr) {
        const int* g = a.groups + blockIdx.x * rt::G_INTS;
        row = g[rt::G_ROW], n = g[rt::G_N], slot = g[rt::G_SLOT];
    } else {
        row = blockIdx.x, slot = a.slots[row];
    }
    const int back = blockIdx.y;
    if (back >= n) return;
    row += n - 1 - back;
    const T* src = (const T*)a.z + row * a.ldz + a.zx;
    T* dst = (T*)a.tail + ((long long)slot * a.ring + a.pos[row] % a.ring) * ch;
    for (int c = threadIdx.x * 4; c < ch; c += CT * 4) store4(dst + c, load4(src + c));
}

template <typename T>
static int launch_conv(const Args& a, cudaStream_t st) {
    const dim3 grid((a.rows + CROWS - 1) / CROWS, (a.channels() / 4 + CT - 1) / CT);
    if (a.taps == 4) ssd_conv_kernel<T, 4><<<grid, CT, 0, st>>>(a);
    else ssd_conv_kernel<T, 0><<<grid, CT, 0, st>>>(a);
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess || a.tail == nullptr) return (int)e;
    ssd_tail_kernel<T><<<dim3(a.groups != nullptr ? a.n : a.rows, a.taps), CT, 0, st>>>(a);
    return (int)cudaGetLastError();
}

// -------------------------------------------------------------------------------------------------------- prompts: recurrence
constexpr int RT = 256, COLS = 64, TOK = 16, LD = COLS + 8;

// grid (requests, H, column slices of 64).  Thread 4 j + r owns rows r mod 4 of column j of the state, which lies in shared memory.
template <typename T>
__global__ void __launch_bounds__(RT) ssd_scan_kernel(Args a) {
    extern __shared__ float sm[];
    const int dn = a.dn, dv = a.dv;
    float* S = sm;                       // [dn][COLS + 8]
    float* C = S + dn * LD;              // [TOK][dn]
    float* B = C + TOK * dn;             // [TOK][dn]
    float* X = B + TOK * dn;             // [TOK][COLS]
    __shared__ float dt[TOK], decay[TOK];
    const int h = blockIdx.y, g = h / (a.H / a.G), c0 = blockIdx.z * COLS, nc = min(COLS, dv - c0);
    int row0 = blockIdx.x, n = 1, slot, flags;
    if (a.groups != nullptr) {
        const int* it = a.groups + blockIdx.x * rt::G_INTS;
        row0 = it[rt::G_ROW], n = it[rt::G_N], slot = it[rt::G_SLOT], flags = it[rt::G_FLAGS];
    } else {                             // one token per request, positions only known here
        slot = a.slots[row0], flags = a.pos[row0] > 0 ? 7 : 3;
    }
    float* state = a.state == nullptr ? nullptr : a.state + ((long long)slot * a.H + h) * dn * dv;
    for (int i = threadIdx.x; i < dn * COLS; i += RT) {
        const int r = i / COLS, c = i % COLS;
        S[r * LD + c] = (flags & 4) && state != nullptr && c < nc ? state[(long long)r * dv + c0 + c] : 0.f;
    }
    const float D = a.d[h];
    const int j = threadIdx.x >> 2, part = threadIdx.x & 3;
    for (int t0 = 0; t0 < n; t0 += TOK) {
        const int nt = min(TOK, n - t0);
        __syncthreads();
        for (int i = threadIdx.x; i < nt * dn; i += RT) {
            const T* p = (const T*)a.xbc + (long long)(row0 + t0 + i / dn) * a.ldx + a.H * dv + g * dn + i % dn;
            B[i] = to_f(p[0]);
            C[i] = to_f(p[a.G * dn]);
        }
        for (int i = threadIdx.x; i < nt * COLS; i += RT)
            X[i] = i % COLS < nc ? to_f(((const T*)a.xbc)[(long long)(row0 + t0 + i / COLS) * a.ldx + h * dv + c0 + i % COLS]) : 0.f;
        if (threadIdx.x < nt) {
            const long long i = (long long)(row0 + t0 + threadIdx.x) * a.H + h;
            dt[threadIdx.x] = a.dt[i];
            decay[threadIdx.x] = expf(a.la[i]);
        }
        __syncthreads();
        for (int t = 0; t < nt; ++t) {
            const float x = X[t * COLS + j], in = dt[t] * x, f = decay[t];
            float o = 0.f;
            for (int r = part; r < dn; r += 4) {
                const float s = f * S[r * LD + j] + B[t * dn + r] * in;
                S[r * LD + j] = s;
                o += C[t * dn + r] * s;
            }
            o += __shfl_xor_sync(0xffffffffu, o, 1);
            o += __shfl_xor_sync(0xffffffffu, o, 2);
            if (part == 0 && j < nc) ((float*)a.y)[(row0 + t0 + t) * a.ldy + h * dv + c0 + j] = o + D * x;
        }
    }
    __syncthreads();
    if (state != nullptr)
        for (int i = threadIdx.x; i < dn * nc; i += RT) state[(long long)(i / nc) * dv + c0 + i % nc] = S[i / nc * LD + i % nc];
}

template <typename T>
static int launch_scan(const Args& a, cudaStream_t st) {
    const size_t smem = sizeof(float) * ((size_t)a.dn * LD + 2 * TOK * a.dn + TOK * COLS);
    if (smem > 226 * 1024) return -2;
    cudaError_t e = cudaFuncSetAttribute(ssd_scan_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    ssd_scan_kernel<T><<<dim3(a.groups != nullptr ? a.n : a.rows, a.H, (a.dv + COLS - 1) / COLS), RT, smem, st>>>(a);
    return (int)cudaGetLastError();
}

// ---------------------------------------------------------------------------------------------------------------- one token
constexpr int ST = 256, SW = ST / 32;

// How a CTA goes over a state: a thread owns 4 columns and every `parts`-th row, `slots` of them.
struct StepShape {
    int cols, parts, slots, partial;     // partial: rows of partial sums over the state's rows that meet in shared memory
    __host__ __device__ StepShape(int dn, int dv) {
        cols = dv / 4, parts = ST / cols, slots = (dn + parts - 1) / parts;
        partial = 32 % cols == 0 ? SW : parts;               // (threads of a warp that share columns add up among themselves)
    }
    __host__ __device__ int stage() const { return slots * ST * 16; }
    __host__ __device__ int rest(int dn, int dv, int heads) const { return 4 * (heads * dv + 2 * dn + 2 * partial * dv); }
};

// grid (H / heads, n): `heads` heads of one group, one after the other; while one is worked on, the next one's state is on its way into
// shared memory (every thread waits for its own pieces only).
template <typename T>
__global__ void __launch_bounds__(ST, 3) ssd_step_kernel(Args a, int heads) {
    extern __shared__ float4 sm4[];
    const int h0 = blockIdx.x * heads, b = blockIdx.y, dn = a.dn, dv = a.dv, g = h0 / (a.H / a.G), ch = a.channels();
    const StepShape sh(dn, dv);
    const int c = threadIdx.x % sh.cols * 4, r0 = threadIdx.x / sh.cols, warp = threadIdx.x >> 5, stages = heads > 1 ? 2 : 1;
    float4* stage = sm4 + threadIdx.x;                       // [stages][slots][ST]
    float* X = reinterpret_cast<float*>(sm4 + stages * sh.slots * ST);   // [heads][dv]
    float* B = X + heads * dv;                               // [dn]
    float* C = B + dn;                                       // [dn]
    float* O = C + dn;                                       // [2][partial][dv]
    const bool on = r0 < sh.parts;
    // slots and positions, the state and the convolution's past are older than the kernel before this one
    const int pos = a.pos[b], slot = a.slots[b];
    const bool fresh = pos == 0;
    float* S = a.state + ((long long)slot * a.H + h0) * dn * dv;
    auto fetch = [&](int i) {                                // head h0 + i
        if (i < heads && on && !fresh) {
            const float* p = S + (long long)i * dn * dv;
            for (int k = 0, r = r0; r < dn; ++k, r += sh.parts)
                cp_async16(stage + ((i & (stages - 1)) * sh.slots + k) * ST, p + (long long)r * dv + c, true);
        }
        cp_async_commit();
    };
    fetch(0);
    T* tail = (T*)a.tail + (long long)slot * a.ring * ch;
    const int back = min(a.taps - 1, pos), own = heads * dv; // inputs the convolution sees besides the token's own
    auto channel = [&](int i) { return i < own ? h0 * dv + i : i < own + dn ? a.H * dv + g * dn + i - own : a.H * dv + (a.G + g) * dn + i - own - dn; };
    auto older = [&](int k) {
        float v = a.conv_bias[k];
        for (int n = back; n > 0; --n) v += a.conv[(long long)(a.taps - 1 - n) * ch + k] * to_f(tail[(long long)((pos - n) % a.ring) * ch + k]);
        return v;
    };
    const int numbers = own + 2 * dn;
    float pre[2];                                            // what they add up to for this thread's first channels
    pre[0] = threadIdx.x < numbers ? older(channel(threadIdx.x)) : 0.f;
    pre[1] = threadIdx.x + ST < numbers ? older(channel(threadIdx.x + ST)) : 0.f;
    pdl_trigger();
    asm volatile("griddepcontrol.wait;" ::: "memory");
    const T* z = (const T*)a.z + (long long)b * a.ldz;
    for (int i = threadIdx.x, n = 0; i < numbers; i += ST, ++n) {
        const int k = channel(i);
        const T x = z[a.zx + k];
        const float v = (n == 0 ? pre[0] : n == 1 ? pre[1] : older(k)) + a.conv[(long long)(a.taps - 1) * ch + k] * to_f(x);
        X[i] = to_f(from_f<T>(silu<T>(v)));
        // a ring of `taps` rows: the place of this input is none that another CTA still reads
        if (i < own || h0 % (a.H / a.G) == 0) tail[(long long)(pos % a.ring) * ch + k] = x;
    }
    __syncthreads();
    for (int i = 0; i < heads; ++i) {
        const int h = h0 + i;
        if (stages > 1) fetch(i + 1);
        const float dt = softplus(to_f(z[a.zdt + h]) + a.dt_bias[h]), decay = expf(-expf(a.a_log[h]) * dt);
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f), o = v;
        if (on) v = load4(X + i * dv + c);
        v = make_float4(v.x * dt, v.y * dt, v.z * dt, v.w * dt);
        if (stages > 1) cp_async_wait<1>();
        else cp_async_wait<0>();
        if (on) {
            const float4* from = stage + (i & (stages - 1)) * sh.slots * ST;
            float* to = S + (long long)i * dn * dv + c;
#pragma unroll 8
            for (int k = 0; k < sh.slots; ++k) {
                const int r = r0 + k * sh.parts;
                if (r < dn) {
                    float4 s = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : from[k * ST];
                    const float in = B[r], q = C[r];
                    s = make_float4(decay * s.x + in * v.x, decay * s.y + in * v.y, decay * s.z + in * v.z, decay * s.w + in * v.w);
                    *reinterpret_cast<float4*>(to + (long long)r * dv) = s;
                    o.x += q * s.x; o.y += q * s.y; o.z += q * s.z; o.w += q * s.w;
                }
            }
        }
        bool writes = on;
        int at = r0;
        if (sh.partial == SW && 32 % sh.cols == 0) {
            for (int k = sh.cols; k < 32; k <<= 1) {
                o.x += __shfl_xor_sync(0xffffffffu, o.x, k); o.y += __shfl_xor_sync(0xffffffffu, o.y, k);
                o.z += __shfl_xor_sync(0xffffffffu, o.z, k); o.w += __shfl_xor_sync(0xffffffffu, o.w, k);
            }
            writes = (threadIdx.x & 31) < sh.cols;
            at = warp;
        }
        float* part = O + (i & 1) * sh.partial * dv;
        if (writes) *reinterpret_cast<float4*>(part + at * dv + c) = o;
        __syncthreads();
        if (threadIdx.x < dv) {                              // dv <= ST: a thread finishes one column
            float y = a.d[h] * X[i * dv + threadIdx.x];
            for (int r = 0; r < sh.partial; ++r) y += part[r * dv + threadIdx.x];
            ((float*)a.y)[b * a.ldy + h * dv + threadIdx.x] = y;
        }
    }
}

template <typename T>
static int launch_step(const Args& a, int sms, cudaStream_t st) {
    const StepShape sh(a.dn, a.dv);
    // several heads per CTA once there are more CTAs than fit the GPU at a time
    int heads = 1;
    const int each = a.H / a.G;
    while (each % (2 * heads) == 0 && (long long)a.H * a.n >= 6LL * heads * sms && 2 * sh.stage() + sh.rest(a.dn, a.dv, 2 * heads) <= 74 * 1024) heads *= 2;
    const int smem = (heads > 1 ? 2 : 1) * sh.stage() + sh.rest(a.dn, a.dv, heads);
    if (smem > 220 * 1024) return -2;
    cudaError_t e = cudaFuncSetAttribute(ssd_step_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return (int)e;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(a.H / heads, a.n);
    cfg.blockDim = dim3(ST);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    return (int)cudaLaunchKernelEx(&cfg, ssd_step_kernel<T>, a, heads);
}

// ------------------------------------------------------------------------------------------------------------- gate and norm
constexpr int NT = 256, NW = NT / 32, KEEP = 4;

// A CTA is a row.  Up to 8 norm groups share its warps evenly, more groups take turns on single warps.  Numbers of a group are counted
// without padding: number i is column i % nv of head i / nv.  V divides nv and the group's size.
template <typename Y, typename T, int V>
__global__ void __launch_bounds__(NT) ssd_norm_kernel(Args a) {
    pdl_trigger();
    __shared__ float red[NW];
    const int w = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int size = a.H * a.nv / a.norm_groups, share = a.norm_groups < NW ? NW / a.norm_groups : 1;
    const int part = w % share, step = share * 32 * V, row = blockIdx.x;
    const Y* y = (const Y*)a.y + row * a.ldy;
    const T* z = (const T*)a.z + row * a.ldz + a.zz;
    T* out = (T*)a.out + row * a.ldo;
    for (int g0 = 0; g0 < a.norm_groups; g0 += NW / share) {
        const int g = g0 + w / share, lo = g * size, hi = g < a.norm_groups ? lo + size : lo;
        const int at = lo + (part * 32 + lane) * V;
        float x[KEEP][V];
        auto place = [&](int i) { return a.nv == a.dv ? i : i / a.nv * a.dv + i % a.nv; };
        auto gated = [&](int i, float (&v)[V]) {
            const int c = place(i);
            float f[V], q[V];
            if constexpr (V == 4) {
                const float4 s = load4(y + c), t = load4(z + c);
                f[0] = s.x, f[1] = s.y, f[2] = s.z, f[3] = s.w;
                q[0] = t.x, q[1] = t.y, q[2] = t.z, q[3] = t.w;
            } else {
                f[0] = to_f(y[c]), q[0] = to_f(z[c]);
            }
#pragma unroll
            for (int e = 0; e < V; ++e) v[e] = f[e] * silu<T>(q[e]);
        };
        float s = 0.f;
#pragma unroll
        for (int k = 0; k < KEEP; ++k) {
            if (at + k * step < hi) {
                gated(at + k * step, x[k]);
#pragma unroll
                for (int e = 0; e < V; ++e) s += x[k][e] * x[k][e];
            }
        }
        for (int i = at + KEEP * step; i < hi; i += step) {
            float v[V];
            gated(i, v);
#pragma unroll
            for (int e = 0; e < V; ++e) s += v[e] * v[e];
        }
        s = warp_sum(s);
        if (share > 1) {                                     // (then there is one turn)
            if (lane == 0) red[w] = s;
            __syncthreads();
            s = 0.f;
            for (int i = 0; i < share; ++i) s += red[min(w / share * share + i, NW - 1)];
        }
        const float r = a.mul / sqrtf(s / size + a.eps);
        auto finish = [&](int i, const float (&v)[V]) {
            const int c = place(i);
            if constexpr (V == 4) {
                const float4 k = load4(a.norm + c);
                store4(out + c, make_float4(v[0] * r * k.x, v[1] * r * k.y, v[2] * r * k.z, v[3] * r * k.w));
            } else {
                out[c] = from_f<T>(v[0] * r * a.norm[c]);
            }
        };
#pragma unroll
        for (int k = 0; k < KEEP; ++k)
            if (at + k * step < hi) finish(at + k * step, x[k]);
        for (int i = at + KEEP * step; i < hi; i += step) {
            float v[V];
            gated(i, v);
            finish(i, v);
        }
    }
    if (a.nv < a.dv)                                         // columns between the heads
        for (int i = threadIdx.x; i < a.H * (a.dv - a.nv); i += NT) out[i / (a.dv - a.nv) * a.dv + a.nv + i % (a.dv - a.nv)] = from_f<T>(0.f);
}

template <typename Y, typename T>
static int launch_norm(const Args& a, cudaStream_t st) {
    if (a.nv % 4 == 0 && a.H * a.nv / a.norm_groups % 4 == 0) ssd_norm_kernel<Y, T, 4><<<a.rows, NT, 0, st>>>(a);
    else ssd_norm_kernel<Y, T, 1><<<a.rows, NT, 0, st>>>(a);
    return (int)cudaGetLastError();
}

static bool aligned(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }
static bool ok(const Args& a, int dt) {
    const int w = dt ? 8 : 4;
    return a.rows > 0 && a.H > 0 && a.G > 0 && a.H % a.G == 0 && a.dn > 0 && a.dv > 0 && a.dn % 16 == 0 && a.dv % 16 == 0 && a.nv > 0 && a.nv <= a.dv && a.taps > 0 &&
           a.taps <= MAX_TAPS && a.ldz % w == 0 && a.ldo % w == 0 && a.ldy % 8 == 0 && a.zz % w == 0 && a.zx % w == 0 && a.norm_groups > 0 &&
           a.H * a.nv % a.norm_groups == 0 && (a.tail == nullptr || a.ring >= a.taps) && aligned(a.z) && aligned(a.state) && aligned(a.tail) && aligned(a.y) &&
           aligned(a.conv) && aligned(a.conv_bias) && aligned(a.norm) && aligned(a.out);
}

}  // namespace ssd
}  // namespace lmoe

using namespace lmoe;

// z -> xbc, dt, la; then the tails of the requests (groups: whole requests; null: one row each).  dt: 1 bf16, 0 fp32
LMOE_API int lmoe_ssd_conv(const ssd::Args* ap, int dt, cudaStream_t st) {
    const ssd::Args& a = *ap;
    if (!ssd::ok(a, dt) || a.xbc == nullptr || a.dt == nullptr || a.la == nullptr || a.ldx % 8 || (a.groups != nullptr && a.n <= 0)) return -1;
    return dt ? ssd::launch_conv<bf16>(a, st) : ssd::launch_conv<float>(a, st);
}

// Groups that are whole requests (flags 3 or 7), or (a.groups null) one token per request; y fp32
LMOE_API int lmoe_ssd_scan(const ssd::Args* ap, int dt, cudaStream_t st) {
    const ssd::Args& a = *ap;
    if (!ssd::ok(a, dt) || !a.y_f32 || a.xbc == nullptr || a.dt == nullptr || a.la == nullptr || (a.groups != nullptr && a.n <= 0)) return -1;
    return dt ? ssd::launch_scan<bf16>(a, st) : ssd::launch_scan<float>(a, st);
}

// One token per request, state and tail in place, y fp32: dv <= 256, a state of up to 192 KB; rows with position 0 start from zero.  Slots and positions must have been
// on the device before the kernel that precedes this one in the stream was launched.
LMOE_API int lmoe_ssd_step(const ssd::Args* ap, int dt, int sms, cudaStream_t st) {
    const ssd::Args& a = *ap;
    if (sms <= 0 || !ssd::ok(a, dt) || a.n != a.rows || a.dv > 256 || a.state == nullptr || a.tail == nullptr || !a.y_f32) return -1;
    return dt ? ssd::launch_step<bf16>(a, sms, st) : ssd::launch_step<float>(a, sms, st);
}

// y, z -> out
LMOE_API int lmoe_ssd_norm(const ssd::Args* ap, int dt, cudaStream_t st) {
    const ssd::Args& a = *ap;
    if (!ssd::ok(a, dt)) return -1;
    if (!dt) return a.y_f32 ? ssd::launch_norm<float, float>(a, st) : -1;
    return a.y_f32 ? ssd::launch_norm<float, bf16>(a, st) : ssd::launch_norm<bf16, bf16>(a, st);
}
