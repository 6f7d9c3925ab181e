// Row kernels of blocks that norm both ends of a sublayer, x += mul post(f(pre(x))), around an fp32 residual stream:
//   residual_norm   y = the sublayer's output rows (or the sum of a token's expert rows, and of another row);  x += mul y / rms(y) * post;
//                   h = x / rms(x) * pre, the input of the next sublayer: one pass over the stream per sublayer
//   glu_rows        silu(gate) * up, or relu(gate) * up
//   xielu_rows      a0 z^2 + z / 2 for positive z, else a1 (e^z - 1 - z) + z / 2, in place
// Rows are padded to a multiple of 4 elements (pad = 0).  Compiled without fast-math: the same code serves the fp32 model.
#include "common.cuh"

namespace lmoe {
namespace sb {

constexpr int THREADS = 256, NV = 4;         // float4s a thread keeps in registers (rows up to 4096 wide)

__device__ __forceinline__ float dot4(float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
__device__ __forceinline__ float4 mul4(float4 v, float r, float4 w) { return make_float4(v.x * r * w.x, v.y * r * w.y, v.z * r * w.z, v.w * r * w.w); }
__device__ __forceinline__ float4 add4(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }

// top > 0: y holds one row per (token, expert); those of token t are rows dest[t * top + k] (dest null: t * top + k).  plus: one more row per
// token (null: none)
template <typename Y, typename T>
__global__ void __launch_bounds__(THREADS) residual_norm_kernel(float* __restrict__ x, long long ldx, const Y* __restrict__ y, long long ldy,
                                                                const int* __restrict__ dest, int top, const Y* __restrict__ plus, long long ldp,
                                                                float mul, const float* __restrict__ post, const float* __restrict__ pre, T* __restrict__ h, long long ldh, int width,
                                                                int pad, float eps) {
    pdl_trigger();
    __shared__ float red[32];
    float* xr = x + (long long)blockIdx.x * ldx;
    auto load_y = [&](int c) {
        float4 s = plus == nullptr ? make_float4(0.f, 0.f, 0.f, 0.f) : load4(plus + (long long)blockIdx.x * ldp + c);
        if (top <= 0) return add4(s, load4(y + (long long)blockIdx.x * ldy + c));
        for (int k = 0; k < top; ++k) {
            const long long i = (long long)blockIdx.x * top + k;
            s = add4(s, load4(y + (dest == nullptr ? i : (long long)dest[i]) * ldy + c));
        }
        return s;
    };
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    float4 v[NV], xv[NV];
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = (threadIdx.x + i * THREADS) * 4;
        xv[i] = c < pad ? load4(xr + c) : zero;
        v[i] = c < pad ? load_y(c) : zero;
        s += dot4(v[i]);
    }
    for (int c = (threadIdx.x + NV * THREADS) * 4; c < pad; c += THREADS * 4) s += dot4(load_y(c));
    const float ry = mul / sqrtf(block_sum(s, red) / width + eps);
    s = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = (threadIdx.x + i * THREADS) * 4;
        if (c < pad) {
            xv[i] = add4(xv[i], mul4(v[i], ry, load4(post + c)));
            store4(xr + c, xv[i]);
            s += dot4(xv[i]);
        }
    }
    for (int c = (threadIdx.x + NV * THREADS) * 4; c < pad; c += THREADS * 4) {
        const float4 t = add4(load4(xr + c), mul4(load_y(c), ry, load4(post + c)));
        store4(xr + c, t);
        s += dot4(t);
    }
    if (pre == nullptr) return;
    const float rx = 1.f / sqrtf(block_sum(s, red) / width + eps);
    T* hr = h + (long long)blockIdx.x * ldh;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = (threadIdx.x + i * THREADS) * 4;
        if (c < pad) store4(hr + c, mul4(xv[i], rx, load4(pre + c)));
    }
    for (int c = (threadIdx.x + NV * THREADS) * 4; c < pad; c += THREADS * 4) store4(hr + c, mul4(load4(xr + c), rx, load4(pre + c)));
}

// z [rows, ldz]: gate in columns 0 .. ff, up in ff .. 2 ff
template <typename T>
__global__ void __launch_bounds__(THREADS) glu_rows_kernel(const T* __restrict__ z, long long ldz, T* __restrict__ out, long long ldo, int ff, int relu) {
    pdl_trigger();
    constexpr int W = Vec<T>::N;
    const T* zr = z + (long long)blockIdx.x * ldz;
    T* o = out + (long long)blockIdx.x * ldo;
    for (int c = (threadIdx.x + blockIdx.y * THREADS) * W; c < ff; c += gridDim.y * THREADS * W) {
        Vec<T> g, u;
        g.load(zr + c);
        u.load(zr + ff + c);
#pragma unroll
        for (int i = 0; i < W; ++i) {
            const float t = g.get(i);
            g.set(i, (relu ? fmaxf(t, 0.f) : t / (1.f + expf(-t))) * u.get(i));
        }
        g.store(o + c);
    }
}

template <typename T>
__global__ void __launch_bounds__(THREADS) xielu_rows_kernel(T* __restrict__ z, long long ldz, int cols, const float* __restrict__ act) {
    pdl_trigger();
    constexpr int W = Vec<T>::N;
    T* zr = z + (long long)blockIdx.x * ldz;
    const float a0 = act[0], a1 = act[1];
    for (int c = (threadIdx.x + blockIdx.y * THREADS) * W; c < cols; c += gridDim.y * THREADS * W) {
        Vec<T> v;
        v.load(zr + c);
#pragma unroll
        for (int i = 0; i < W; ++i) {
            const float t = v.get(i);
            v.set(i, (t > 0.f ? a0 * t * t : a1 * (expm1f(t) - t)) + 0.5f * t);
        }
        v.store(zr + c);
    }
}

template <typename Y, typename T>
static int launch(float* x, long long ldx, const void* y, long long ldy, const int* dest, int top, const void* plus, long long ldp, float mul,
                  const float* post, const float* pre, void* h, long long ldh, int rows, int width, int pad, float eps, cudaStream_t st) {
    residual_norm_kernel<Y, T><<<rows, THREADS, 0, st>>>(x, ldx, (const Y*)y, ldy, dest, top, (const Y*)plus, ldp, mul, post, pre, (T*)h, ldh, width, pad, eps);
    return (int)cudaGetLastError();
}

}  // namespace sb
}  // namespace lmoe

using namespace lmoe;

// y_dt, dt: 1 bf16, 0 fp32 (of y and h).  pad: columns of x, h, post and pre (a multiple of 4, zeros from width on); y has at least pad
// columns with zeros from width on, and so has plus (y's type).
LMOE_API int lmoe_residual_norm(float* x, long long ldx, const void* y, long long ldy, int y_dt, const int* dest, int top, const void* plus,
                                long long ldp, float mul, const float* post, const float* pre, void* h, long long ldh, int rows, int width, int pad, float eps, int dt, cudaStream_t st) {
    if (rows <= 0 || width <= 0 || pad < width || pad % 4 || ldx % 4 || ldy % 4 || ldp % 4 || (pre != nullptr && ldh % 4)) return -1;
    if (y_dt) return dt ? sb::launch<bf16, bf16>(x, ldx, y, ldy, dest, top, plus, ldp, mul, post, pre, h, ldh, rows, width, pad, eps, st)
                        : sb::launch<bf16, float>(x, ldx, y, ldy, dest, top, plus, ldp, mul, post, pre, h, ldh, rows, width, pad, eps, st);
    return dt ? sb::launch<float, bf16>(x, ldx, y, ldy, dest, top, plus, ldp, mul, post, pre, h, ldh, rows, width, pad, eps, st)
              : sb::launch<float, float>(x, ldx, y, ldy, dest, top, plus, ldp, mul, post, pre, h, ldh, rows, width, pad, eps, st);
}

// kind: 0 silu, 1 relu
LMOE_API int lmoe_glu_rows(const void* z, long long ldz, void* out, long long ldo, int rows, int ff, int kind, int dt, cudaStream_t st) {
    const int w = dt ? 8 : 4;
    if (kind < 0 || kind > 1 || rows <= 0 || ff <= 0 || ff % w || ldz % w || ldo % w || ((reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(out)) & 15)) return -1;
    int cols = (ff + sb::THREADS * w - 1) / (sb::THREADS * w);
    if (rows > 1024) cols = 1;
    if (dt) sb::glu_rows_kernel<bf16><<<dim3(rows, cols), sb::THREADS, 0, st>>>((const bf16*)z, ldz, (bf16*)out, ldo, ff, kind);
    else sb::glu_rows_kernel<float><<<dim3(rows, cols), sb::THREADS, 0, st>>>((const float*)z, ldz, (float*)out, ldo, ff, kind);
    return (int)cudaGetLastError();
}

// act: {a0, a1}
LMOE_API int lmoe_xielu_rows(void* z, long long ldz, int rows, int cols, const float* act, int dt, cudaStream_t st) {
    const int w = dt ? 8 : 4;
    if (rows <= 0 || cols <= 0 || cols % w || ldz % w || act == nullptr || (reinterpret_cast<uintptr_t>(z) & 15)) return -1;
    const int parts = rows > 1024 ? 1 : (cols + sb::THREADS * w - 1) / (sb::THREADS * w);
    if (dt) sb::xielu_rows_kernel<bf16><<<dim3(rows, parts), sb::THREADS, 0, st>>>((bf16*)z, ldz, cols, act);
    else sb::xielu_rows_kernel<float><<<dim3(rows, parts), sb::THREADS, 0, st>>>((float*)z, ldz, cols, act);
    return (int)cudaGetLastError();
}
