// Arguments of the state-space kernels (ssd*.cu); groups and requests are tables of retention.cuh.
#pragma once
#include "retention.cuh"

namespace lmoe {
namespace ssd {

constexpr int MAX_TAPS = 16;             // of the convolution

struct Args {
    const void* z;                       // [rows, ldz]: z (H x dv) from column zz; x (H x dv), B, C (G x dn each) from column zx; dt (H) from column zdt
    void* xbc;                           // [rows, ldx]: x, B, C behind the convolution
    float *dt, *la;                      // [rows, H] step sizes, log decays
    void *y, *out;                       // [rows, ldy]: H x dv, fp32 (y_f32) or bf16; [rows, ldo]: H x dv
    const float *conv, *conv_bias;       // [taps, channels], [channels]
    const float *dt_bias, *a_log, *d;    // [H]
    const float* norm;                   // [H * dv]
    void* tail;                          // [slots, ring, channels] inputs of the convolution, row = position modulo ring, or null
    float* state;                        // [slots, H, dn, dv] or null
    float *scratch, *decay;              // [places, H, dn, dv]; [places, H]: log decay of the group in front of the place
    const int *pos, *slots;              // [rows]
    const int *groups, *requests;        // [n, 8], [m, 8]
    long long ldz, ldx, ldy, ldo;
    int zz, zx, zdt, H, G, dn, dv;       // head sizes as laid out
    int nv;                              // a head's columns without padding
    int taps, ring, rows, n, m, norm_groups, y_f32;
    float mul, eps;
    __host__ __device__ int channels() const { return H * dv + 2 * G * dn; }
};

}  // namespace ssd
}  // namespace lmoe
