// What the scans of the matrix-state recurrences share: small asynchronous copies into shared memory and the
// butterfly that sums many values over a warp's lanes at once.
#pragma once

#include "common.cuh"

namespace llmb {

__device__ __forceinline__ void copy4(float* smem, const float* global) {
    unsigned s = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(s), "l"(global));
}
__device__ __forceinline__ void copy16(float* smem, const float* global) {
    unsigned s = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(s), "l"(global));
}
__device__ __forceinline__ void copies_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int LEFT> __device__ __forceinline__ void copies_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(LEFT)); }

// One level of a butterfly over COUNT values a lane: lanes whose bit OFFSET is set keep the upper half of the
// values and hand over the lower half, the others the reverse; what stays is own + partner's. After the
// levels 16, 8, 4, 2, 1 on 32 values lane l holds the sum over all lanes of value l. Every value's sum runs through
// the same tree of lane pairs (l, l ^ 16), then (l, l ^ 8), ..., whatever its index: a sum does not depend on the
// place of its token in a group.
template <int COUNT, int OFFSET, int SIZE>
__device__ __forceinline__ void fold(float (&v)[SIZE], int lane) {
    bool up = (lane & OFFSET) != 0;
#pragma unroll
    for (int k = 0; k < COUNT; ++k) {
        float send = up ? v[k] : v[COUNT + k];
        float keep = up ? v[COUNT + k] : v[k];
        v[k] = keep + __shfl_xor_sync(0xffffffffu, send, OFFSET);
    }
}

}  // namespace llmb
