// Arguments of the chunked-attention kernels.
#pragma once
namespace lmoe {
// one work item of the prompt kernels: eight int32
enum {
    I_ROW,       // packed row of the item's first query
    I_NQ,        // queries
    I_C0,        // place of the first query in its chunk
    I_FRESH0,    // place in the chunk of the first key that is in this call (earlier ones are in the cache)
    I_SLOT,      // cache slot of the request
    I_N = 8
};

namespace ca {
struct Args {
    const void* z;            // [rows, ldz] projection output
    void* out;                // [rows, ldo]
    void *kc, *vc;            // cache [slots, cap_rows, G, dkp] / [slots, cap_rows, G, dvp]
    const float* lut;         // [H, nlut] bias by distance (the last entry holds for everything beyond)
    const float* gain;        // 1 float
    const int* items;         // rows kernel: [n, 8] work items
    const int* slots;         // step: [B]; store: [rows]
    const int* pos;           // step: [B]; store: [rows] position of the token
    const int* ends;          // store: [rows] length of the token's request after this call
    long long ldz, ldo;
    int zq, zk, zv, zg;       // first columns
    int H, G, dk, dv, dkp, dvp;
    int cap_rows, size, nlut;
    int n;                    // work items / requests / rows
    float scale, cap, mul;
};
}  // namespace ca
}  // namespace lmoe
