// Arguments of the generalized delta rule's kernels (delta_rule*.cu); groups are tables of retention.cuh.
#pragma once
#include "retention.cuh"

namespace lmoe {
namespace dlt {

constexpr float DECAY = 0.60653065971263342f;               // exp(-1/2): a channel's log decay is -DECAY sigmoid(.)
constexpr float UNIT_EPS = 1e-6f;                            // in the length of a key

struct Args {
    const void* z;                       // [rows, ldz]: r, k, v, removal rate, gate (H x d each)
    void* out;                           // [rows, ldo]: H x d
    const float* w;                      // [rows, ldw]: second projection of the decay
    const float *w0, *a_bias, *norm;     // [H * d]
    float* state;                        // [slots, H, d, d] or null
    float* raw;                          // general kernel: [rows, H * d]
    void* work;                          // tensor-core kernels: what the chunks leave for the pass over them
    const int *pos, *slots;              // [rows]
    const int* groups;                   // [n, 8]
    long long ldz, ldo, ldw;
    int zr, zk, zv, za, zg, H, d;
    int nd;                              // a head's numbers without padding
    int rows, n;
    float eps;
};

}  // namespace dlt
}  // namespace lmoe
