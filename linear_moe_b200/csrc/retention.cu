// Retention, S <- decay S + k v^T, o = scale S^T q, out = o / rms(o) * silu(gate), head by head with an fp32 state per request:
//   retention_step_kernel   one token per request: rotation, state update, norm and gate in one pass over the state (bf16 or fp32)
//   retention_rows_kernel   prompts of any head size, bf16 or fp32, token by token in fp32 (bf16 fast path: retention_tc.cu), and
//   norm_gate_kernel        the norm and gate behind it
// Compiled without fast-math: the fp32 instantiations serve models in true 32-bit.
#include "common.cuh"
#include "retention.cuh"

namespace lmoe {
namespace rt {

// ---------------------------------------------------------------------------------------------------------------- one token
constexpr int ST = 512;

// grid (H, n).  A thread owns 4 columns of the state and every `parts`-th row (parts = ST / (dv / 4)), NB of them in flight.
template <typename T>
__global__ void __launch_bounds__(ST, 2) retention_step_kernel(Args a) {
    constexpr int NB = 8;
    extern __shared__ float4 sm4[];
    const int h = blockIdx.x, b = blockIdx.y, dk = a.dk, dv = a.dv, half = a.rot / 2;
    const int cols = dv / 4, parts = ST / cols, c = threadIdx.x % cols * 4, r0 = threadIdx.x / cols;
    float* O = reinterpret_cast<float*>(sm4);                // [parts][dv]
    float* Q = O + parts * dv;                               // [dk]
    float* K = Q + dk;                                       // [dk]
    __shared__ float red[32];
    const bool on = r0 < parts;
    const bool fresh = a.pos[b] == 0;
    float* S = a.state + ((long long)a.slots[b] * a.H + h) * dk * dv;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    // the state is older than the kernel before this one
    float4 s[NB];
#pragma unroll
    for (int i = 0; i < NB; ++i) {
        const int r = r0 + i * parts;
        s[i] = on && r < dk && !fresh ? *reinterpret_cast<const float4*>(S + (long long)r * dv + c) : zero;
    }
    pdl_trigger();
    asm volatile("griddepcontrol.wait;" ::: "memory");
    const T* z = (const T*)a.z + (long long)b * a.ldz;
    for (int d = threadIdx.x; d < dk; d += ST) {
        const T *q = z + a.zq + h * dk, *k = z + a.zk + h * dk;
        float x = to_f(q[d]), y = to_f(k[d]);
        if (d < a.rot) {
            const bool low = d < half;
            const int o = low ? d + half : d - half;
            const float2 cs = a.turn[(long long)b * half + (low ? d : o)];
            const float xo = to_f(q[o]), yo = to_f(k[o]);
            x = low ? x * cs.x - xo * cs.y : x * cs.x + xo * cs.y;
            y = low ? y * cs.x - yo * cs.y : y * cs.x + yo * cs.y;
        }
        Q[d] = x * a.scale;
        K[d] = y;
    }
    float4 v = zero, o = zero;
    if (on) v = load4(z + a.zv + h * dv + c);
    const float decay = (float)a.decay[h];
    __syncthreads();
    for (int rb = r0; on && rb < dk; rb += NB * parts) {
#pragma unroll
        for (int i = 0; i < NB; ++i) {
            const int r = rb + i * parts;
            if (r < dk) {
                const float k = K[r], q = Q[r];
                s[i].x = decay * s[i].x + k * v.x; s[i].y = decay * s[i].y + k * v.y;
                s[i].z = decay * s[i].z + k * v.z; s[i].w = decay * s[i].w + k * v.w;
                *reinterpret_cast<float4*>(S + (long long)r * dv + c) = s[i];
                o.x += q * s[i].x; o.y += q * s[i].y; o.z += q * s[i].z; o.w += q * s[i].w;
            }
        }
#pragma unroll
        for (int i = 0; i < NB; ++i) {
            const int r = rb + (NB + i) * parts;
            if (r < dk) s[i] = fresh ? zero : *reinterpret_cast<const float4*>(S + (long long)r * dv + c);
        }
    }
    if (on) *reinterpret_cast<float4*>(O + r0 * dv + c) = o;
    __syncthreads();
    float y = 0.f;                                           // dv <= ST: a thread finishes one column
    if (threadIdx.x < dv)
        for (int r = 0; r < parts; ++r) y += O[r * dv + threadIdx.x];
    const float rms = 1.f / sqrtf(block_sum(y * y, red) / a.nv + a.eps);
    if (threadIdx.x < dv) {
        const float g = to_f(z[a.zg + h * dv + threadIdx.x]);
        ((T*)a.out)[(long long)b * a.ldo + h * dv + threadIdx.x] = from_f<T>(y * rms * (g / (1.f + expf(-g))));
    }
}

template <typename T>
static int launch_step(const Args& a, cudaStream_t st) {
    const size_t smem = sizeof(float) * (2 * a.dk + ST / (a.dv / 4) * a.dv);
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
    return (int)cudaLaunchKernelEx(&cfg, retention_step_kernel<T>, a);
}

// ------------------------------------------------------------------------------------------------------------------ prompts
constexpr int RT = 256, COLS = 64, TOK = 16, LD = COLS + 8;

// grid (groups, H, column slices of 64).  Thread 4 j + r owns rows r mod 4 of column j of the state, which lies in shared memory.
template <typename T>
__global__ void __launch_bounds__(RT) retention_rows_kernel(Args a) {
    extern __shared__ float sm[];
    const int dk = a.dk, dv = a.dv;
    float* S = sm;                       // [dk][COLS + 8]
    float* Q = S + dk * LD;              // [TOK][dk]
    float* K = Q + TOK * dk;             // [TOK][dk]
    float* V = K + TOK * dk;             // [TOK][COLS]
    const int h = blockIdx.y, c0 = blockIdx.z * COLS, nc = min(COLS, dv - c0);
    int row0 = blockIdx.x, n = 1, slot, flags;
    if (a.groups != nullptr) {
        const int* g = a.groups + blockIdx.x * G_INTS;
        row0 = g[G_ROW], n = g[G_N], slot = g[G_SLOT], flags = g[G_FLAGS];
    } else {                             // one token per request, positions only known here
        slot = a.slots[row0], flags = a.pos[row0] > 0 ? 7 : 3;
    }
    float* state = a.state == nullptr ? nullptr : a.state + ((long long)slot * a.H + h) * dk * dv;
    for (int i = threadIdx.x; i < dk * COLS; i += RT) {
        const int r = i / COLS, c = i % COLS;
        S[r * LD + c] = (flags & 4) && state != nullptr && c < nc ? state[(long long)r * dv + c0 + c] : 0.f;
    }
    const float decay = (float)a.decay[h];
    const int j = threadIdx.x >> 2, part = threadIdx.x & 3;
    for (int t0 = 0; t0 < n; t0 += TOK) {
        const int nt = min(TOK, n - t0);
        __syncthreads();
        for (int i = threadIdx.x; i < nt * dk; i += RT) {
            const T* z = (const T*)a.z + (long long)(row0 + t0 + i / dk) * a.ldz + h * dk + i % dk;
            Q[i] = to_f(z[a.zq]);
            K[i] = to_f(z[a.zk]);
        }
        for (int i = threadIdx.x; i < nt * COLS; i += RT)
            V[i] = i % COLS < nc ? to_f(((const T*)a.z)[(long long)(row0 + t0 + i / COLS) * a.ldz + a.zv + h * dv + c0 + i % COLS]) : 0.f;
        __syncthreads();
        for (int t = 0; t < nt; ++t) {
            const float v = V[t * COLS + j];
            float o = 0.f;
            for (int r = part; r < dk; r += 4) {
                const float s = decay * S[r * LD + j] + K[t * dk + r] * v;
                S[r * LD + j] = s;
                o += Q[t * dk + r] * s;
            }
            o += __shfl_xor_sync(0xffffffffu, o, 1);
            o += __shfl_xor_sync(0xffffffffu, o, 2);
            if (part == 0 && j < nc) a.raw[((long long)(row0 + t0 + t) * a.H + h) * dv + c0 + j] = o * a.scale;
        }
    }
    __syncthreads();
    if (state != nullptr)
        for (int i = threadIdx.x; i < dk * nc; i += RT) state[(long long)(i / nc) * dv + c0 + i % nc] = S[i / nc * LD + i % nc];
}

// one warp per (row, head)
template <typename T>
__global__ void __launch_bounds__(256) norm_gate_kernel(Args a) {
    const long long i = blockIdx.x * 8LL + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31, h = (int)(i % a.H);
    const long long row = i / a.H;
    if (row >= a.m) return;
    const float* o = a.raw + (row * a.H + h) * a.dv;
    float s = 0.f;
    for (int d = lane; d < a.dv; d += 32) s += o[d] * o[d];
    const float r = 1.f / sqrtf(warp_sum(s) / a.nv + a.eps);
    const T* g = (const T*)a.z + row * a.ldz + a.zg + h * a.dv;
    for (int d = lane; d < a.dv; d += 32) {
        const float x = to_f(g[d]);
        ((T*)a.out)[row * a.ldo + h * a.dv + d] = from_f<T>(o[d] * r * (x / (1.f + expf(-x))));
    }
}

template <typename T>
static int launch_rows(const Args& a, cudaStream_t st) {
    const size_t smem = sizeof(float) * ((size_t)a.dk * LD + 2 * TOK * a.dk + TOK * COLS);
    if (smem > 227 * 1024) return -2;
    cudaError_t e = cudaFuncSetAttribute(retention_rows_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    retention_rows_kernel<T><<<dim3(a.n, a.H, (a.dv + COLS - 1) / COLS), RT, smem, st>>>(a);
    if ((e = cudaGetLastError()) != cudaSuccess) return (int)e;
    norm_gate_kernel<T><<<(unsigned)(((long long)a.m * a.H + 7) / 8), 256, 0, st>>>(a);
    return (int)cudaGetLastError();
}

static bool ok(const Args& a, int dt) {
    const int w = dt ? 8 : 4;
    return a.n > 0 && a.H > 0 && a.dk > 0 && a.dv > 0 && a.dk % 16 == 0 && a.dv % 16 == 0 && a.nv > 0 && a.rot >= 0 && a.rot % 2 == 0 && a.rot <= a.dk &&
           a.ldz % w == 0 && a.ldo % w == 0 && a.decay != nullptr && ((reinterpret_cast<uintptr_t>(a.z) | reinterpret_cast<uintptr_t>(a.state)) & 15) == 0;
}

}  // namespace rt
}  // namespace lmoe

using namespace lmoe;

// One token per request, state in place: a.state, dv <= 256; rows with position 0 start from zero.  Slots and positions must have been on
// the device before the kernel that precedes this one in the stream was launched.
LMOE_API int lmoe_retention_step(const rt::Args* ap, int dt, cudaStream_t st) {
    const rt::Args& a = *ap;
    if (!rt::ok(a, dt) || a.dv > 256 || a.state == nullptr || (a.rot > 0 && a.turn == nullptr) || a.zq % 4 || a.zk % 4 || a.zv % 4) return -1;
    return dt ? rt::launch_step<bf16>(a, st) : rt::launch_step<float>(a, st);
}

// Groups that are whole requests (flags 3 or 7), or (a.groups null) one token per request; a.raw [m, H * dv], m rows in all.
LMOE_API int lmoe_retention_rows(const rt::Args* ap, int dt, cudaStream_t st) {
    const rt::Args& a = *ap;
    if (!rt::ok(a, dt) || a.m <= 0 || a.raw == nullptr) return -1;
    return dt ? rt::launch_rows<bf16>(a, st) : rt::launch_rows<float>(a, st);
}
