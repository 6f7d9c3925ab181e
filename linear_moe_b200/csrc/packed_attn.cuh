// Arguments of the packed-row attention kernels (packed_attn*.cu).
//
// Queries are rows of one matrix, keys and values rows of two others (column ranges of a projection, or buffers of their own when
// a prompt goes on from a cache).  A cache keeps keys and values as rows [row, kv head, dim] of one buffer, addressed through a
// request's slot in one of two ways:
//   ring   (table null)  row = slot * cap + position % cap: the last `cap` positions, for layers with a window
//   pages  (table)       row = table[slot][position / PAGE] * PAGE + position % PAGE: every position
#pragma once
namespace lmoe {
namespace pa {

constexpr int PAGE = 64;

// one work item of the prompt kernels: eight int32
enum {
    I_ROW,       // row of the item's first query
    I_NQ,        // queries
    I_C0,        // place of the first query among its request's keys
    I_KROW,      // row of the request's first key
    I_N = 8
};

struct Prompt {
    const void *q, *k, *v, *gate;     // gate: null or [rows, ldg], the output is multiplied by its sigmoid
    void* out;                        // [rows, ldo], head by head dv columns
    const int* items;                 // [n, 8]
    int* err;                         // tensor-core kernel: status word of its bounded waits
    long long ldq, ldk, ldv, ldg, ldo;
    int H, G, dk, dv;
    int window;                       // <= 0: none
    int n, q_rows, k_rows;
    float scale;
    int cross;                        // every query head's weights are applied to the values of every kv head: out [rows, H, G, dv]
    int bounded;                      // cross, tensor-core kernel: |q . k * scale| <= 60 everywhere, so that exp needs no running maximum
    const float* bias;                // [H]: weights sigmoid(q . k * scale + bias[h]) that sum to nothing in particular (null: softmax)
    float mul;                        // factor of the output with these
};

struct Cache {
    void *k, *v;                      // [rows, G, dk], [rows, G, dv]
    const int* table;                 // null: ring
    int table_ld, cap;
    __device__ __forceinline__ long long row(int slot, int pos) const {
        return table == nullptr ? (long long)slot * cap + pos % cap : (long long)table[(long long)slot * table_ld + pos / PAGE] * PAGE + pos % PAGE;
    }
};

struct Step {
    const void* q;                    // [n, ldq], head by head dk columns
    void* out;                        // [n, ldo], head by head dv columns
    Cache c;                          // holds the new token's key and value already
    const int *pos, *slots;           // [n] position of the new token, cache slot
    long long ldq, ldo;
    int H, G, dk, dv;
    int window;                       // <= 0: none
    int n;
    float scale;
    int cross;                        // as in Prompt
    const float* bias;                // as in Prompt
    float mul;
};

}  // namespace pa
}  // namespace lmoe
