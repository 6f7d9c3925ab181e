// Arguments of the retention kernels (retention*.cu).
#pragma once
namespace lmoe {
namespace rt {

// a run of a request's new tokens: eight int32
enum {
    G_ROW,       // first row
    G_N,         // tokens
    G_SLOT,
    G_FLAGS,     // 1: the request's first group, 2: its last one, 4: the request has a past
    G_IN,        // place in `scratch` of the state in front of it (-1: the request's own, or zero)
    G_OUT,       // place in `scratch` of the state behind it (-1: none)
    G_INTS = 8
};
// a request of several groups: eight int32 (slot, flags, first place in `scratch`, groups, tokens of all groups but the last)
enum { R_SLOT, R_FLAGS, R_STATE, R_GROUPS, R_TOKENS };

struct Args {
    void *z, *out;                       // [rows, ldz]: queries, keys (H x dk), values, gate (H x dv); [rows, ldo]: H x dv
    float* state;                        // [slots, H, dk, dv] or null
    float* scratch;                      // [places, H, dk, dv]
    float* raw;                          // general kernel: [rows, H * dv]
    const float* powers;                 // [H, 65] decay^0 ..
    const double* decay;                 // [H]
    const float2* turn;                  // [rows, rot / 2] (cos, sin) (one-token kernel; prompts are rotated before)
    const int *pos, *slots;              // [rows]
    const int *groups, *requests;        // [n, 8], [m, 8]
    long long ldz, ldo;
    int zq, zk, zv, zg, H, dk, dv;
    int nv;                              // numbers in the output norm (unpadded)
    int rot, n, m;
    float scale, eps;
};

}  // namespace rt
}  // namespace lmoe
