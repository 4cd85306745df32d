// Greedy pick shared by the heads: (logit, row) candidates, the lowest row on ties, merged over CTAs.
#pragma once
#include "portable.h"

namespace llvq {

constexpr int kHeadThreads = 256;   // 8 warps, one embedding row per warp and step
constexpr int kHeadMaxGrid = 1024;  // partial (value, row) pairs the pick kernel merges
constexpr int kHeadMaxHidden = 8192;

struct HeadBest {
    float val;
    int row;
};

__device__ __forceinline__ bool head_better(float v, int r, float bv, int br) { return v > bv || (v == bv && r < br); }

// One CTA: merge the partials; the row index is reported with `row_offset` added (a vocabulary shard).
__global__ void __launch_bounds__(kHeadMaxGrid)
lm_head_pick_kernel(const HeadBest* __restrict__ partial, int n, long long row_offset, float* __restrict__ val_out,
                    long long* __restrict__ idx_out) {
    llvq_dependent_enter();
    __shared__ HeadBest red[32];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    HeadBest b = threadIdx.x < n ? partial[threadIdx.x] : HeadBest{-INFINITY, 0x7fffffff};
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float v = __shfl_xor_sync(0xffffffffu, b.val, o);
        const int r = __shfl_xor_sync(0xffffffffu, b.row, o);
        if (head_better(v, r, b.val, b.row)) b = HeadBest{v, r};
    }
    if (lane == 0) red[warp] = b;
    __syncthreads();
    if (warp == 0) {
        b = red[lane];
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float v = __shfl_xor_sync(0xffffffffu, b.val, o);
            const int r = __shfl_xor_sync(0xffffffffu, b.row, o);
            if (head_better(v, r, b.val, b.row)) b = HeadBest{v, r};
        }
        if (lane == 0) {
            *val_out = b.val;
            *idx_out = row_offset + (b.row == 0x7fffffff ? 0 : b.row);  // all-NaN logits: row 0
        }
    }
}

}  // namespace llvq
