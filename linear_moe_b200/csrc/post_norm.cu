// Row kernels of blocks that norm a sublayer's output only, x += norm(f(x)) * gain, around an fp32 residual stream; the norm takes its
// root mean square in `groups` equal consecutive parts of a row:
//   residual_group_norm   x += y / rms(y) * gain;  h = x in the model's dtype, the input of the next sublayer: one pass over the stream
//   group_norm            h = x / rms(x) * gain
//   embed_rows            x = embedding[token] in fp32, h = the same in the model's dtype
//   softcap               z = cap tanh(z / cap)
// Rows are padded to a multiple of 4 elements (pad = 0).  Compiled without fast-math: the same code serves the fp32 model.
#include "common.cuh"

namespace lmoe {
namespace pn {

constexpr int THREADS = 256, WARPS = THREADS / 32, NV = 4;

template <int V> struct Num;             // V consecutive numbers
template <> struct Num<4> {
    float4 v;
    template <typename T> __device__ __forceinline__ void load(const T* p) { v = load4(p); }
    template <typename T> __device__ __forceinline__ void store(T* p) const { store4(p, v); }
    __device__ __forceinline__ float square() const { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
    __device__ __forceinline__ void scale(float r, const Num& g) { v = make_float4(v.x * r * g.v.x, v.y * r * g.v.y, v.z * r * g.v.z, v.w * r * g.v.w); }
    __device__ __forceinline__ void add(const Num& o) { v = make_float4(v.x + o.v.x, v.y + o.v.y, v.z + o.v.z, v.w + o.v.w); }
    __device__ __forceinline__ void zero() { v = make_float4(0.f, 0.f, 0.f, 0.f); }
};
template <> struct Num<1> {
    float v;
    template <typename T> __device__ __forceinline__ void load(const T* p) { v = to_f(*p); }
    template <typename T> __device__ __forceinline__ void store(T* p) const { *p = from_f<T>(v); }
    __device__ __forceinline__ float square() const { return v * v; }
    __device__ __forceinline__ void scale(float r, const Num& g) { v = v * r * g.v; }
    __device__ __forceinline__ void add(const Num& o) { v += o.v; }
    __device__ __forceinline__ void zero() { v = 0.f; }
};

// Up to 8 groups share the warps of a CTA (a row) evenly; more groups take turns on single warps.  V divides the group's size.
// RES: x += norm(y) gain, h = x (h null: not wanted).  Else h = norm(y) gain, x unused.
template <typename Y, typename T, int V, bool RES>
__global__ void __launch_bounds__(THREADS) group_norm_kernel(float* __restrict__ x, long long ldx, const Y* __restrict__ y, long long ldy,
                                                             const float* __restrict__ gain, T* __restrict__ h, int width, int pad, int groups, float eps) {
    pdl_trigger();
    __shared__ float red[WARPS];
    const int w = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int size = width / groups, share = groups < WARPS ? WARPS / groups : 1;   // warps of a group
    const int part = w % share, step = share * 32 * V;
    float* xr = x + (long long)blockIdx.x * ldx;
    const Y* yr = y + (long long)blockIdx.x * ldy;
    T* hr = h + (long long)blockIdx.x * pad;
    for (int g0 = 0; g0 < groups; g0 += WARPS / share) {     // more than one turn only where share is 1
        const int g = g0 + w / share, lo = g * size, hi = g < groups ? lo + size : lo;
        const int at = lo + (part * 32 + lane) * V;
        Num<V> v[NV], xv[NV];
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = at + i * step;
            if (RES && c < hi) xv[i].load(xr + c);
            if (c < hi) v[i].load(yr + c);
            else v[i].zero();
        }
#pragma unroll
        for (int i = 0; i < NV; ++i) s += v[i].square();
        for (int c = at + NV * step; c < hi; c += step) {
            Num<V> t;
            t.load(yr + c);
            s += t.square();
        }
        s = warp_sum(s);
        if (share > 1) {
            if (lane == 0) red[w] = s;
            __syncthreads();
            s = 0.f;
            for (int i = 0; i < share; ++i) s += red[min(w / share * share + i, WARPS - 1)];
        }
        const float r = 1.f / sqrtf(s / size + eps);
        auto finish = [&](int c, Num<V> t, const Num<V>& o) {
            Num<V> k;
            k.load(gain + c);
            t.scale(r, k);
            if (RES) {
                t.add(o);
                t.store(xr + c);
            }
            if (h != nullptr) t.store(hr + c);
        };
#pragma unroll
        for (int i = 0; i < NV; ++i)
            if (at + i * step < hi) finish(at + i * step, v[i], xv[i]);
        for (int c = at + NV * step; c < hi; c += step) {
            Num<V> t, o;
            t.load(yr + c);
            if (RES) o.load(xr + c);
            finish(c, t, o);
        }
    }
    if (h != nullptr)
        for (int c = width + threadIdx.x; c < pad; c += THREADS) hr[c] = from_f<T>(0.f);
}

template <typename Y, typename T, bool RES>
static int launch(float* x, long long ldx, const void* y, long long ldy, const float* gain, void* h, int rows, int width, int pad, int groups, float eps,
                  cudaStream_t st) {
    if (width / groups % 4 == 0) group_norm_kernel<Y, T, 4, RES><<<rows, THREADS, 0, st>>>(x, ldx, (const Y*)y, ldy, gain, (T*)h, width, pad, groups, eps);
    else group_norm_kernel<Y, T, 1, RES><<<rows, THREADS, 0, st>>>(x, ldx, (const Y*)y, ldy, gain, (T*)h, width, pad, groups, eps);
    return (int)cudaGetLastError();
}

template <typename T>
__global__ void __launch_bounds__(THREADS) embed_rows_kernel(const long long* __restrict__ ids, const T* __restrict__ emb, float* __restrict__ x,
                                                             T* __restrict__ h, int width, int pad, int vocab) {
    pdl_trigger();
    // ids are checked on the host; the clamp keeps a bad one from becoming a bad address
    const T* e = emb + min(max(ids[blockIdx.x], 0LL), (long long)vocab - 1) * width;
    float* xr = x + (long long)blockIdx.x * pad;
    T* hr = h + (long long)blockIdx.x * pad;
    for (int c = threadIdx.x; c < pad; c += THREADS) {
        const T v = c < width ? e[c] : from_f<T>(0.f);
        xr[c] = to_f(v);
        hr[c] = v;
    }
}

__global__ void __launch_bounds__(THREADS) softcap_kernel(float* z, long long n, float cap) {
    for (long long i = blockIdx.x * (long long)THREADS + threadIdx.x; i < n; i += (long long)gridDim.x * THREADS) z[i] = cap * tanhf(z[i] / cap);
}

static bool aligned(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }
static bool shape_ok(int rows, int width, int pad, int groups) { return rows > 0 && width > 0 && pad >= width && pad % 4 == 0 && groups > 0 && width % groups == 0; }

}  // namespace pn
}  // namespace lmoe

using namespace lmoe;

// y_dt, dt: 1 bf16, 0 fp32 (of y and h).  x [rows, ldx], gain [pad], h [rows, pad] or null; pad a multiple of 4, x and gain zero from
// width on; y has at least width columns; 16-byte bases, pitches multiples of 4.
LMOE_API int lmoe_residual_group_norm(float* x, long long ldx, const void* y, long long ldy, int y_dt, const float* gain, void* h, int rows, int width,
                                      int pad, int groups, float eps, int dt, cudaStream_t st) {
    if (!pn::shape_ok(rows, width, pad, groups) || ldx % 4 || ldy % 4 || !pn::aligned(x) || !pn::aligned(y) || !pn::aligned(gain) || !pn::aligned(h)) return -1;
    if (y_dt) return dt ? pn::launch<bf16, bf16, true>(x, ldx, y, ldy, gain, h, rows, width, pad, groups, eps, st)
                        : pn::launch<bf16, float, true>(x, ldx, y, ldy, gain, h, rows, width, pad, groups, eps, st);
    return dt ? pn::launch<float, bf16, true>(x, ldx, y, ldy, gain, h, rows, width, pad, groups, eps, st)
              : pn::launch<float, float, true>(x, ldx, y, ldy, gain, h, rows, width, pad, groups, eps, st);
}

LMOE_API int lmoe_group_norm(const float* x, long long ldx, const float* gain, void* h, int rows, int width, int pad, int groups, float eps, int dt,
                             cudaStream_t st) {
    if (!pn::shape_ok(rows, width, pad, groups) || ldx % 4 || h == nullptr || !pn::aligned(x) || !pn::aligned(gain) || !pn::aligned(h)) return -1;
    return dt ? pn::launch<float, bf16, false>(nullptr, 0, x, ldx, gain, h, rows, width, pad, groups, eps, st)
              : pn::launch<float, float, false>(nullptr, 0, x, ldx, gain, h, rows, width, pad, groups, eps, st);
}

LMOE_API int lmoe_embed_rows(const long long* ids, const void* emb, float* x, void* h, int rows, int width, int pad, int vocab, int dt, cudaStream_t st) {
    if (rows <= 0 || width <= 0 || pad < width || vocab <= 0) return -1;
    if (dt) pn::embed_rows_kernel<bf16><<<rows, pn::THREADS, 0, st>>>(ids, (const bf16*)emb, x, (bf16*)h, width, pad, vocab);
    else pn::embed_rows_kernel<float><<<rows, pn::THREADS, 0, st>>>(ids, (const float*)emb, x, (float*)h, width, pad, vocab);
    return (int)cudaGetLastError();
}

LMOE_API int lmoe_softcap(float* z, long long n, float cap, cudaStream_t st) {
    if (n <= 0 || !(cap > 0.f)) return -1;
    const long long blocks = (n + pn::THREADS - 1) / pn::THREADS;
    pn::softcap_kernel<<<(unsigned)(blocks < 148 * 16 ? blocks : 148 * 16), pn::THREADS, 0, st>>>(z, n, cap);
    return (int)cudaGetLastError();
}
