// Generalized delta rule over packed rows, head by head in fp32,
//     S <- diag(w) S - (a u)(u^T S) + k v^T,    o = S^T r,    out = o / rms(o) * weight * sigmoid(gate)
// with the unit key u, decays w = exp(-DECAY sigmoid(W2 tanh(.) + w0)) and rates a = sigmoid(. + bias) per channel:
//   delta_low_kernel    tanh of the decay's inner activations (the second projection is a matrix product), or for few rows in bf16
//   delta_decay_kernel  both
//   delta_rows_kernel   prompts of any size, bf16 or fp32, token by token (bf16 fast path: delta_rule_tc.cu), and
//   delta_norm_kernel   the norm and gate behind it
//   delta_step_kernel   one token per request, everything else in one pass over the state
// With the old state S, p = S^T u and q = S^T (w r), the output is o = q - (r . a u) p + (r . k) v: one reduction over the rows of S.
// Compiled without fast-math: the fp32 instantiations serve models in true 32-bit.
#include "delta_rule.cuh"
#include "mma_utils.cuh"

namespace lmoe {
namespace dlt {

__device__ __forceinline__ float sigmoid(float x) { return 1.f / (1.f + expf(-x)); }

template <typename T>
__global__ void __launch_bounds__(256) delta_low_kernel(const T* __restrict__ z, long long ldz, T* __restrict__ low, long long ldl, int rows, int cols) {
    pdl_trigger();
    const long long total = (long long)rows * (cols / 4);
    for (long long i = blockIdx.x * 256LL + threadIdx.x; i < total; i += gridDim.x * 256LL) {
        const long long row = i / (cols / 4);
        const int c = (int)(i - row * (cols / 4)) * 4;
        const float4 x = load4(z + row * ldz + c);
        store4(low + row * ldl + c, make_float4(tanhf(x.x), tanhf(x.y), tanhf(x.z), tanhf(x.w)));
    }
}

// Few rows, bf16: tanh and the second projection in one launch.  A CTA has 64 channels, a warp 16 of them; grid (channels / 64 rounded up).
constexpr int DR = 64;                   // rows at most

__global__ void __launch_bounds__(128) delta_decay_kernel(const bf16* __restrict__ z, long long ldz, const bf16* __restrict__ w2, float* __restrict__ out,
                                                          int rows, int rank, int channels) {
    extern __shared__ __align__(16) unsigned char smem[];
    const int ld = rank + 8, c0 = blockIdx.x * 64, w = threadIdx.x >> 5, l = threadIdx.x & 31, g = l >> 2, q = l & 3;
    bf16* W = reinterpret_cast<bf16*>(smem);                 // [64][ld]
    bf16* L = W + 64 * ld;                                   // [rows up to the next 16][ld]
    for (int i = threadIdx.x; i < 64 * (rank / 8); i += 128) {           // (weights do not change)
        const int r = i / (rank / 8), c = i % (rank / 8) * 8;
        cp_async16(W + r * ld + c, w2 + (c0 + r < channels ? (long long)(c0 + r) * rank + c : 0), c0 + r < channels);
    }
    cp_async_commit();
    pdl_trigger();
    asm volatile("griddepcontrol.wait;" ::: "memory");
    const int tiles = (rows + 15) / 16;
    for (int i = threadIdx.x; i < tiles * 16 * (rank / 4); i += 128) {
        const int r = i / (rank / 4), c = i % (rank / 4) * 4;
        const float4 x = r < rows ? load4(z + r * ldz + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        store4(L + r * ld + c, make_float4(tanhf(x.x), tanhf(x.y), tanhf(x.z), tanhf(x.w)));
    }
    cp_async_wait<0>();
    __syncthreads();
    float acc[DR / 8][4];
    zero_acc<DR / 8>(acc);
    for (int k0 = 0; k0 < rank; k0 += 16) {
        uint32_t p[4];
        load_a(p, W, ld, 16 * w, k0);
#pragma unroll
        for (int t = 0; t < DR / 16; ++t)
            if (t < tiles) {
                uint32_t b[4];
                load_b2(b, L, ld, 16 * t, k0);
                mma16816(acc[2 * t], p, b[0], b[1]);
                mma16816(acc[2 * t + 1], p, b[2], b[3]);
            }
    }
#pragma unroll
    for (int t = 0; t < DR / 8; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int r = 8 * t + 2 * q + (e & 1), c = c0 + 16 * w + g + 8 * (e >> 1);
            if (r < rows && c < channels) out[(long long)r * channels + c] = acc[t][e];
        }
}

// ------------------------------------------------------------------------------------------------------------------ prompts
constexpr int RT = 256, COLS = 64, TOK = 16, LD = COLS + 8;

// grid (requests, H, column slices of 64).  Thread 4 j + r owns rows r mod 4 of column j of the state, which lies in shared memory.
template <typename T>
__global__ void __launch_bounds__(RT) delta_rows_kernel(Args a) {
    extern __shared__ float sm[];
    const int d = a.d;
    float* S = sm;                       // [d][COLS + 8]
    float* R = S + d * LD;               // [TOK][d] each
    float* K = R + TOK * d;
    float* U = K + TOK * d;
    float* A = U + TOK * d;              // a u
    float* W = A + TOK * d;
    float* V = W + TOK * d;              // [TOK][COLS]
    const int h = blockIdx.y, c0 = blockIdx.z * COLS, nc = min(COLS, d - c0);
    int row0 = blockIdx.x, n = 1, slot, flags;
    if (a.groups != nullptr) {
        const int* g = a.groups + blockIdx.x * rt::G_INTS;
        row0 = g[rt::G_ROW], n = g[rt::G_N], slot = g[rt::G_SLOT], flags = g[rt::G_FLAGS];
    } else {                             // one token per request, positions only known here
        slot = a.slots[row0], flags = a.pos[row0] > 0 ? 7 : 3;
    }
    float* state = a.state == nullptr ? nullptr : a.state + ((long long)slot * a.H + h) * d * d;
    for (int i = threadIdx.x; i < d * COLS; i += RT) {
        const int r = i / COLS, c = i % COLS;
        S[r * LD + c] = (flags & 4) && state != nullptr && c < nc ? state[(long long)r * d + c0 + c] : 0.f;
    }
    const int j = threadIdx.x >> 2, part = threadIdx.x & 3, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int t0 = 0; t0 < n; t0 += TOK) {
        const int nt = min(TOK, n - t0);
        __syncthreads();
        for (int t = warp; t < nt; t += RT / 32) {           // a warp prepares a token
            const long long row = row0 + t0 + t;
            const T* z = (const T*)a.z + row * a.ldz + h * d;
            float s = 0.f;
            for (int c = lane; c < d; c += 32) {
                const float k = to_f(z[a.zk + c]);
                s += k * k;
            }
            const float inv = 1.f / sqrtf(warp_sum(s) + UNIT_EPS);
            for (int c = lane; c < d; c += 32) {
                const float k = to_f(z[a.zk + c]), u = k * inv;
                R[t * d + c] = to_f(z[a.zr + c]);
                K[t * d + c] = k;
                U[t * d + c] = u;
                A[t * d + c] = u * sigmoid(to_f(z[a.za + c]) + a.a_bias[h * d + c]);
                W[t * d + c] = expf(-DECAY * sigmoid(a.w[row * a.ldw + h * d + c] + a.w0[h * d + c]));
            }
        }
        for (int i = threadIdx.x; i < nt * COLS; i += RT)
            V[i] = i % COLS < nc ? to_f(((const T*)a.z)[(long long)(row0 + t0 + i / COLS) * a.ldz + a.zv + h * d + c0 + i % COLS]) : 0.f;
        __syncthreads();
        for (int t = 0; t < nt; ++t) {
            const float v = V[t * COLS + j];
            float p = 0.f, o = 0.f;
            for (int r = part; r < d; r += 4) p += U[t * d + r] * S[r * LD + j];
            p += __shfl_xor_sync(0xffffffffu, p, 1);
            p += __shfl_xor_sync(0xffffffffu, p, 2);
            for (int r = part; r < d; r += 4) {
                const float s = W[t * d + r] * S[r * LD + j] - A[t * d + r] * p + K[t * d + r] * v;
                S[r * LD + j] = s;
                o += R[t * d + r] * s;
            }
            o += __shfl_xor_sync(0xffffffffu, o, 1);
            o += __shfl_xor_sync(0xffffffffu, o, 2);
            if (part == 0 && j < nc) a.raw[((long long)(row0 + t0 + t) * a.H + h) * d + c0 + j] = o;
        }
    }
    __syncthreads();
    if (state != nullptr)
        for (int i = threadIdx.x; i < d * nc; i += RT) state[(long long)(i / nc) * d + c0 + i % nc] = S[i / nc * LD + i % nc];
}

// one warp per (row, head)
template <typename T>
__global__ void __launch_bounds__(256) delta_norm_kernel(Args a) {
    const long long i = blockIdx.x * 8LL + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31, h = (int)(i % a.H);
    const long long row = i / a.H;
    if (row >= a.rows) return;
    const float* o = a.raw + (row * a.H + h) * a.d;
    float s = 0.f;
    for (int c = lane; c < a.d; c += 32) s += o[c] * o[c];
    const float r = 1.f / sqrtf(warp_sum(s) / a.nd + a.eps);
    const T* g = (const T*)a.z + row * a.ldz + a.zg + h * a.d;
    for (int c = lane; c < a.d; c += 32) ((T*)a.out)[row * a.ldo + h * a.d + c] = from_f<T>(o[c] * r * a.norm[h * a.d + c] * sigmoid(to_f(g[c])));
}

template <typename T>
static int launch_rows(const Args& a, cudaStream_t st) {
    const size_t smem = sizeof(float) * ((size_t)a.d * LD + 5 * TOK * a.d + TOK * COLS);
    if (smem > 227 * 1024) return -2;
    cudaError_t e = cudaFuncSetAttribute(delta_rows_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    delta_rows_kernel<T><<<dim3(a.n, a.H, (a.d + COLS - 1) / COLS), RT, smem, st>>>(a);
    if ((e = cudaGetLastError()) != cudaSuccess) return (int)e;
    delta_norm_kernel<T><<<(unsigned)(((long long)a.rows * a.H + 7) / 8), 256, 0, st>>>(a);
    return (int)cudaGetLastError();
}

// ---------------------------------------------------------------------------------------------------------------- one token
// grid (H, n).  A thread owns 4 columns of the state and every `parts`-th row (parts = ST / (d / 4)); the first NB of them stay in registers
// between the reduction and the update.
template <typename T, int ST>
__global__ void __launch_bounds__(ST, ST == 256 ? 5 : 2) delta_step_kernel(Args a) {
    constexpr int NB = ST == 256 ? 4 : 8, NW = ST / 32;
    extern __shared__ float4 sm4[];
    const int h = blockIdx.x, b = blockIdx.y, d = a.d, i = threadIdx.x;
    const int cols = d / 4, parts = ST / cols, c = i % cols * 4, r0 = i / cols, warp = i >> 5, lane = i & 31;
    const bool pairs = 32 % cols == 0;                       // threads of a warp that share columns add up among themselves
    const int partial = pairs ? NW : parts;
    float* P = reinterpret_cast<float*>(sm4);                // [partial][d] partial p
    float* Q = P + partial * d;                              // [partial][d] partial q
    float* U = Q + partial * d;                              // [d] u
    float* F = U + d;                                        // [d] w r
    float* W = F + d;                                        // [d]
    float* A = W + d;                                        // [d] a k (a u without the key's length)
    float* K = A + d;                                        // [d]
    float* Ps = K + d;                                       // [d] p
    __shared__ float red[4][NW];
    const bool on = r0 < parts;
    // the state is older than the kernel before this one
    const bool fresh = a.pos[b] == 0;
    float* S = a.state + ((long long)a.slots[b] * a.H + h) * d * d;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    float4 s[NB];
#pragma unroll
    for (int k = 0; k < NB; ++k) {
        const int r = r0 + k * parts;
        s[k] = on && r < d && !fresh ? *reinterpret_cast<const float4*>(S + (long long)r * d + c) : zero;
    }
    pdl_trigger();
    asm volatile("griddepcontrol.wait;" ::: "memory");
    const T* z = (const T*)a.z + (long long)b * a.ldz + h * d;
    float kk = 0.f, ra = 0.f, rk = 0.f, v = 0.f, gate = 0.f; // d <= ST: a thread has one channel
    if (i < d) {
        const float k = to_f(z[a.zk + i]), r = to_f(z[a.zr + i]), m = sigmoid(to_f(z[a.za + i]) + a.a_bias[h * d + i]) * k;
        const float w = expf(-DECAY * sigmoid(a.w[(long long)b * a.ldw + h * d + i] + a.w0[h * d + i]));
        v = to_f(z[a.zv + i]);
        gate = a.norm[h * d + i] * sigmoid(to_f(z[a.zg + i]));
        U[i] = K[i] = k;
        F[i] = w * r;
        W[i] = w;
        A[i] = m;
        kk = k * k, ra = r * m, rk = r * k;
    }
    if (warp * 32 < d) {
        kk = warp_sum(kk), ra = warp_sum(ra), rk = warp_sum(rk);
        if (lane == 0) red[0][warp] = kk, red[1][warp] = ra, red[2][warp] = rk;
    }
    __syncthreads();
    kk = ra = rk = 0.f;
    for (int k = 0; k * 32 < d; ++k) kk += red[0][k], ra += red[1][k], rk += red[2][k];
    const float inv = 1.f / sqrtf(kk + UNIT_EPS);
    // with p of the key as it is: u = inv k, so p_u = inv p and a u p_u = inv^2 (a k) p
    float4 p = zero, q = zero;
    auto gather = [&](float4 x, int r) {
        const float u = U[r], f = F[r];
        p.x += u * x.x; p.y += u * x.y; p.z += u * x.z; p.w += u * x.w;
        q.x += f * x.x; q.y += f * x.y; q.z += f * x.z; q.w += f * x.w;
    };
    if (on) {
#pragma unroll
        for (int k = 0; k < NB; ++k)
            if (r0 + k * parts < d) gather(s[k], r0 + k * parts);
        if (!fresh)
            for (int r = r0 + NB * parts; r < d; r += parts) gather(*reinterpret_cast<const float4*>(S + (long long)r * d + c), r);
    }
    if (pairs)
        for (int k = cols; k < 32; k <<= 1) {
            p.x += __shfl_xor_sync(0xffffffffu, p.x, k); p.y += __shfl_xor_sync(0xffffffffu, p.y, k);
            p.z += __shfl_xor_sync(0xffffffffu, p.z, k); p.w += __shfl_xor_sync(0xffffffffu, p.w, k);
            q.x += __shfl_xor_sync(0xffffffffu, q.x, k); q.y += __shfl_xor_sync(0xffffffffu, q.y, k);
            q.z += __shfl_xor_sync(0xffffffffu, q.z, k); q.w += __shfl_xor_sync(0xffffffffu, q.w, k);
        }
    if (pairs ? lane < cols : on) {
        *reinterpret_cast<float4*>(P + (pairs ? warp : r0) * d + c) = p;
        *reinterpret_cast<float4*>(Q + (pairs ? warp : r0) * d + c) = q;
    }
    __syncthreads();
    float y = 0.f;
    if (warp * 32 < d) {
        if (i < d) {                                         // this thread's column
            float ps = 0.f, qs = 0.f;
            for (int r = 0; r < partial; ++r) ps += P[r * d + i], qs += Q[r * d + i];
            ps *= inv * inv;
            y = qs - ra * ps + rk * v;
            Ps[i] = ps;
        }
        const float s2 = warp_sum(y * y);
        if (lane == 0) red[3][warp] = s2;
    }
    __syncthreads();
    if (i < d) {
        float s2 = 0.f;
        for (int k = 0; k * 32 < d; ++k) s2 += red[3][k];
        ((T*)a.out)[(long long)b * a.ldo + h * d + i] = from_f<T>(y / sqrtf(s2 / a.nd + a.eps) * gate);
    }
    if (!on) return;
    p = *reinterpret_cast<const float4*>(Ps + c);
    const float4 vs = load4(z + a.zv + c);
    auto update = [&](float4 x, int r) {
        const float w = W[r], m = A[r], k = K[r];
        x = make_float4(w * x.x - m * p.x + k * vs.x, w * x.y - m * p.y + k * vs.y, w * x.z - m * p.z + k * vs.z, w * x.w - m * p.w + k * vs.w);
        *reinterpret_cast<float4*>(S + (long long)r * d + c) = x;
    };
#pragma unroll
    for (int k = 0; k < NB; ++k)
        if (r0 + k * parts < d) update(s[k], r0 + k * parts);
    for (int r = r0 + NB * parts; r < d; r += parts) update(fresh ? zero : *reinterpret_cast<const float4*>(S + (long long)r * d + c), r);
}

template <typename T, int ST>
static int launch_step(const Args& a, cudaStream_t st) {
    const int cols = a.d / 4, partial = 32 % cols == 0 ? ST / 32 : ST / cols;
    const size_t smem = sizeof(float) * (2 * partial + 6) * a.d;
    if (smem > 46 * 1024) return -2;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(a.H, a.n);
    cfg.blockDim = dim3(ST);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    return (int)cudaLaunchKernelEx(&cfg, delta_step_kernel<T, ST>, a);
}

static bool aligned(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }
static bool ok(const Args& a, int dt) {
    const int w = dt ? 8 : 4;
    return a.rows > 0 && a.H > 0 && a.d > 0 && a.d % 16 == 0 && a.nd > 0 && a.nd <= a.d && a.ldz % w == 0 && a.ldo % w == 0 &&
           ((a.zr | a.zk | a.zv | a.za | a.zg) & 7) == 0 && aligned(a.z) && aligned(a.out) && aligned(a.state);
}

}  // namespace dlt
}  // namespace lmoe

using namespace lmoe;

// z [rows, ldz] -> low [rows, ldl], cols a multiple of 4; dt: 1 bf16, 0 fp32
LMOE_API int lmoe_delta_low(const void* z, long long ldz, void* low, long long ldl, int rows, int cols, int dt, cudaStream_t st) {
    if (rows <= 0 || cols <= 0 || cols % 4 || ldz % 4 || ldl % 4 || !dlt::aligned(z) || !dlt::aligned(low)) return -1;
    const long long blocks = ((long long)rows * (cols / 4) + 255) / 256;
    const unsigned grid = (unsigned)(blocks < 148 * 16 ? blocks : 148 * 16);
    if (dt) dlt::delta_low_kernel<bf16><<<grid, 256, 0, st>>>((const bf16*)z, ldz, (bf16*)low, ldl, rows, cols);
    else dlt::delta_low_kernel<float><<<grid, 256, 0, st>>>((const float*)z, ldz, (float*)low, ldl, rows, cols);
    return (int)cudaGetLastError();
}

// bf16: z [rows, ldz] (rank columns, a multiple of 32, up to 64 rows), w2 [channels, rank] -> out [rows, channels] fp32
LMOE_API int lmoe_delta_decay(const void* z, long long ldz, const void* w2, float* out, int rows, int rank, int channels, cudaStream_t st) {
    if (rows <= 0 || rows > dlt::DR || rank <= 0 || rank % 32 || channels <= 0 || ldz % 8 || !dlt::aligned(z) || !dlt::aligned(w2)) return -1;
    const int smem = (64 + (rows + 15) / 16 * 16) * (rank + 8) * 2;
    if (smem > 200 * 1024) return -2;
    cudaError_t e = cudaFuncSetAttribute(dlt::delta_decay_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return (int)e;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3((channels + 63) / 64);
    cfg.blockDim = dim3(128);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    return (int)cudaLaunchKernelEx(&cfg, dlt::delta_decay_kernel, (const bf16*)z, ldz, (const bf16*)w2, out, rows, rank, channels);
}

// Groups that are whole requests (flags 3 or 7), or (a.groups null) one token per request; a.w, a.raw
LMOE_API int lmoe_delta_rows(const dlt::Args* ap, int dt, cudaStream_t st) {
    const dlt::Args& a = *ap;
    if (!dlt::ok(a, dt) || a.n <= 0 || a.raw == nullptr || a.w == nullptr) return -1;
    return dt ? dlt::launch_rows<bf16>(a, st) : dlt::launch_rows<float>(a, st);
}

// One token per request, state in place: a.state, d <= 256; rows with position 0 start from zero.  Slots and positions must have been on the
// device before the kernel that precedes this one in the stream was launched.
LMOE_API int lmoe_delta_step(const dlt::Args* ap, int dt, cudaStream_t st) {
    const dlt::Args& a = *ap;
    if (!dlt::ok(a, dt) || a.n != a.rows || a.d > 256 || a.state == nullptr || a.w == nullptr) return -1;
    if (a.d <= 64) return dt ? dlt::launch_step<bf16, 256>(a, st) : dlt::launch_step<float, 256>(a, st);
    return dt ? dlt::launch_step<bf16, 512>(a, st) : dlt::launch_step<float, 512>(a, st);
}
