// Row kernels of blocks whose mixer and feed-forward read the same fp32 residual stream and add into it together:
//   stream_norm        y = x / rms(x) [* gain]: the fp32 stream -> the input of the block's fused projection (bf16 or fp32).  A
//                      one-number norm gain is a scalar on the projection's outputs, so two norms of the same stream
//                      need one pass and one matrix product; the consumers of the projection apply their gain.  A gain with
//                      one number per column (gain_n > 1, padded like x) is applied here.
//   embed_norm         x = embedding[token] [+ position table[position]] [+ a vector], in fp32, together with the first block's norm; or the
//                      same added to x (layers that run again)
//   poly_norm          sum over p = 1, 2, 3 of w_p u^p / rms(u^p), plus w_4 (element-wise powers, rms over the row)
// Rows are padded (stream and activations to a multiple of 32 elements, pad = 0), so that every product is aligned for TMA.
// Compiled without fast-math: the same code serves the fp32 model.
#include "common.cuh"

namespace lmoe {
namespace pb {

constexpr int THREADS = 256;

// x [rows, ldx] fp32, y [rows, ldy]; columns width .. pad of x hold zeros, and y gets zeros there
template <typename T>
__global__ void __launch_bounds__(THREADS) stream_norm_kernel(const float* __restrict__ x, long long ldx, T* __restrict__ y,
                                                              long long ldy, int width, int pad, float eps, const float* gain, int gain_n) {
    pdl_trigger();
    __shared__ float red[32];
    const float* xr = x + (long long)blockIdx.x * ldx;
    T* yr = y + (long long)blockIdx.x * ldy;
    constexpr int NV = 4;                                   // float4s a thread keeps in registers (rows up to 4096 wide)
    float4 v[NV];
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = (threadIdx.x + i * THREADS) * 4;
        v[i] = c < pad ? *reinterpret_cast<const float4*>(xr + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        s += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
    for (int c = (threadIdx.x + NV * THREADS) * 4; c < pad; c += THREADS * 4) {
        const float4 t = *reinterpret_cast<const float4*>(xr + c);
        s += t.x * t.x + t.y * t.y + t.z * t.z + t.w * t.w;
    }
    const float r = (gain_n == 1 ? *gain : 1.f) / sqrtf(block_sum(s, red) / width + eps);
    auto put = [&](int c, float4 t) {
        const float4 g = gain_n > 1 ? *reinterpret_cast<const float4*>(gain + c) : make_float4(1.f, 1.f, 1.f, 1.f);
        store4(yr + c, make_float4(t.x * r * g.x, t.y * r * g.y, t.z * r * g.z, t.w * r * g.w));
    };
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = (threadIdx.x + i * THREADS) * 4;
        if (c < pad) put(c, v[i]);
    }
    for (int c = (threadIdx.x + NV * THREADS) * 4; c < pad; c += THREADS * 4) put(c, *reinterpret_cast<const float4*>(xr + c));
}

template <typename T>
__global__ void __launch_bounds__(THREADS) embed_norm_kernel(const long long* __restrict__ ids, const int* __restrict__ pos,
                                                             const T* __restrict__ emb, const T* __restrict__ ptab, float* __restrict__ x,
                                                             long long ldx, T* __restrict__ y, long long ldy, int width, int pad,
                                                             int vocab, int npos, float eps, const float* gain, const float* shift, int keep) {
    pdl_trigger();
    __shared__ float red[32];
    // ids and positions are checked on the host; the clamp keeps a bad one from becoming a bad address
    const long long id = min(max(ids[blockIdx.x], 0LL), (long long)vocab - 1);
    const T* er = emb == nullptr ? nullptr : emb + id * width;
    const T* pr = ptab == nullptr ? nullptr : ptab + (long long)min(max(pos[blockIdx.x], 0), npos - 1) * width;
    float* xr = x + (long long)blockIdx.x * ldx;
    T* yr = y + (long long)blockIdx.x * ldy;
    float s = 0.f;
    if (width % 4 == 0 && pad <= 4 * 4 * THREADS) {         // rows in registers, four numbers at a time
        constexpr int NV = 4;
        const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
        auto add = [](float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); };
        float4 v[NV], e[NV], h[NV];
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = (threadIdx.x + i * THREADS) * 4;
            v[i] = keep && c < pad ? load4(xr + c) : zero;
            e[i] = er != nullptr && c < width ? load4(er + c) : zero;
            h[i] = shift != nullptr && c < pad ? load4(shift + c) : zero;
            if (pr != nullptr && c < width) e[i] = add(e[i], load4(pr + c));
        }
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = (threadIdx.x + i * THREADS) * 4;
            v[i] = add(add(v[i], e[i]), h[i]);
            if (c < pad) store4(xr + c, v[i]);
            s += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
        }
        const float r = 1.f / sqrtf(block_sum(s, red) / width + eps);
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = (threadIdx.x + i * THREADS) * 4;
            if (c >= pad) continue;
            const float4 g = gain == nullptr ? make_float4(1.f, 1.f, 1.f, 1.f) : load4(gain + c);
            store4(yr + c, make_float4(v[i].x * r * g.x, v[i].y * r * g.y, v[i].z * r * g.z, v[i].w * r * g.w));
        }
        return;
    }
    for (int c = threadIdx.x; c < pad; c += THREADS) {
        float v = keep ? xr[c] : 0.f;
        if (c < width) v += (er == nullptr ? 0.f : to_f(er[c])) + (pr == nullptr ? 0.f : to_f(pr[c]));
        if (shift != nullptr) v += shift[c];
        xr[c] = v;
        s += v * v;
    }
    const float r = 1.f / sqrtf(block_sum(s, red) / width + eps);
    for (int c = threadIdx.x; c < pad; c += THREADS) yr[c] = from_f<T>(gain == nullptr ? xr[c] * r : xr[c] * r * gain[c]);
}

// z [rows, ldz] -> out [rows, ldo]; gain: the norm gain of the projection's input; act = {w_1, w_2, w_3, w_4}; out *= mul.
// Columns ff .. ff_pad of out get zeros.
template <typename T>
__global__ void __launch_bounds__(THREADS) poly_norm_kernel(const T* __restrict__ z, long long ldz, T* __restrict__ out, long long ldo,
                                                            int ff, int ff_pad, const float* __restrict__ gain,
                                                            const float* __restrict__ act, float eps, float mul, int vec) {
    pdl_trigger();
    __shared__ float red[32];
    const T* zr = z + (long long)blockIdx.x * ldz;
    T* orow = out + (long long)blockIdx.x * ldo;
    const float g = *gain;
    constexpr int W = Vec<T>::N;
    float s1 = 0.f, s2 = 0.f, s3 = 0.f;
    auto add = [&](float u) {
        u *= g;
        const float u2 = u * u, u3 = u2 * u;
        s1 += u2;
        s2 += u2 * u2;
        s3 += u3 * u3;
    };
    if (vec) {
        for (int c = threadIdx.x * W; c < ff; c += THREADS * W) {
            Vec<T> v;
            v.load(zr + c);
#pragma unroll
            for (int i = 0; i < W; ++i) add(v.get(i));
        }
    } else {
        for (int c = threadIdx.x; c < ff; c += THREADS) add(to_f(zr[c]));
    }
    const float inv = 1.f / ff;
    const float r1 = act[0] / sqrtf(block_sum(s1, red) * inv + eps);
    const float r2 = act[1] / sqrtf(block_sum(s2, red) * inv + eps);
    const float r3 = act[2] / sqrtf(block_sum(s3, red) * inv + eps);
    const float e = act[3];
    auto f = [&](float u) {
        u *= g;
        return mul * (((r3 * u + r2) * u + r1) * u + e);
    };
    if (vec) {
        for (int c = threadIdx.x * W; c < ff; c += THREADS * W) {
            Vec<T> v, o;
            v.load(zr + c);
#pragma unroll
            for (int i = 0; i < W; ++i) o.set(i, f(v.get(i)));
            o.store(orow + c);
        }
    } else {
        for (int c = threadIdx.x; c < ff; c += THREADS) orow[c] = from_f<T>(f(to_f(zr[c])));
    }
    for (int c = ff + threadIdx.x; c < ff_pad; c += THREADS) orow[c] = from_f<T>(0.f);
}

}  // namespace pb
}  // namespace lmoe

using namespace lmoe;

// x [rows, ldx] fp32 with zeros in columns width .. pad; y bf16 (dt 1) or fp32 (dt 0); pad a multiple of 4, 16-byte rows; gain: null
// (gain_n 0), one float (gain_n 1) or pad floats (gain_n pad)
LMOE_API int lmoe_stream_norm(const float* x, long long ldx, void* y, long long ldy, int rows, int width, int pad, float eps,
                              const float* gain, int gain_n, int dt, cudaStream_t st) {
    if (rows <= 0 || width <= 0 || pad < width || pad % 4 || ldx % 4 || ldy % 4 || (gain_n != 0 && gain_n != 1 && gain_n != pad) ||
        (gain_n != 0) != (gain != nullptr) || (gain_n > 1 && (reinterpret_cast<uintptr_t>(gain) & 15)))
        return -1;
    if (dt) pb::stream_norm_kernel<bf16><<<rows, pb::THREADS, 0, st>>>(x, ldx, (bf16*)y, ldy, width, pad, eps, gain, gain_n);
    else pb::stream_norm_kernel<float><<<rows, pb::THREADS, 0, st>>>(x, ldx, (float*)y, ldy, width, pad, eps, gain, gain_n);
    return (int)cudaGetLastError();
}

// emb [vocab, width] or null, ptab [npos, width] or null, in the model's dtype; ids int64, pos int32; gain, shift [pad] (zeros behind the width) or
// null; keep: added to x
LMOE_API int lmoe_embed_norm(const long long* ids, const int* pos, const void* emb, const void* ptab, float* x, long long ldx, void* y,
                             long long ldy, int rows, int width, int pad, int vocab, int npos, float eps, const float* gain,
                             const float* shift, int keep, int dt, cudaStream_t st) {
    if (rows <= 0 || width <= 0 || pad < width || pad % 4 || ldx % 4 || ldy % 4 || vocab <= 0 || (ptab != nullptr && npos <= 0)) return -1;
    if (dt) pb::embed_norm_kernel<bf16><<<rows, pb::THREADS, 0, st>>>(ids, pos, (const bf16*)emb, (const bf16*)ptab, x, ldx, (bf16*)y,
                                                                      ldy, width, pad, vocab, npos, eps, gain, shift, keep);
    else pb::embed_norm_kernel<float><<<rows, pb::THREADS, 0, st>>>(ids, pos, (const float*)emb, (const float*)ptab, x, ldx, (float*)y,
                                                                    ldy, width, pad, vocab, npos, eps, gain, shift, keep);
    return (int)cudaGetLastError();
}

LMOE_API int lmoe_poly_norm(const void* z, long long ldz, void* out, long long ldo, int rows, int ff, int ff_pad, const float* gain,
                            const float* act, float eps, float mul, int dt, cudaStream_t st) {
    if (rows <= 0 || ff <= 0 || ff_pad < ff) return -1;
    const int w = dt ? 8 : 4;
    const int vec = ff % w == 0 && ldz % w == 0 && ldo % w == 0 &&
                    ((reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
    if (dt) pb::poly_norm_kernel<bf16><<<rows, pb::THREADS, 0, st>>>((const bf16*)z, ldz, (bf16*)out, ldo, ff, ff_pad, gain, act, eps, mul, vec);
    else pb::poly_norm_kernel<float><<<rows, pb::THREADS, 0, st>>>((const float*)z, ldz, (float*)out, ldo, ff, ff_pad, gain, act, eps, mul, vec);
    return (int)cudaGetLastError();
}
