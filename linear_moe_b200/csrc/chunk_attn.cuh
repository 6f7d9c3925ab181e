// One work item of the chunked-attention prompt kernels: eight int32.
#pragma once
namespace lmoe {
enum {
    I_ROW,       // packed row of the item's first query
    I_NQ,        // queries
    I_C0,        // place of the first query in its chunk
    I_FRESH0,    // place in the chunk of the first key that is in this call (earlier ones are in the cache)
    I_SLOT,      // cache slot of the request
    I_N = 8
};
}  // namespace lmoe
