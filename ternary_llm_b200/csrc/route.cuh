// The choice of a token's experts from the router's logits.
#pragma once
#include <cfloat>
#include <climits>

namespace tllm {

// One warp: the `top` largest of z[0..experts) in order and the softmax over them; idx, wgt in
// shared memory.  Lane l looks at entries l, l + 32, ...
__device__ __forceinline__ void choose_experts(const float* z, int experts, int top, int* idx, float* wgt)
{
    const int lane = threadIdx.x & 31;
    float last = FLT_MAX, first = 0.f;
    int last_i = -1;
    for (int s = 0; s < top; s++) {
        // the largest entry behind (last, last_i) in the order (value down, index up)
        float best = -FLT_MAX;
        int bi = INT_MAX;
        for (int i = lane; i < experts; i += 32) {
            const float v = fminf(fmaxf(z[i], -FLT_MAX), FLT_MAX);    // a NaN goes to the end
            const bool behind = v < last || (v == last && i > last_i);
            if (behind && (bi == INT_MAX || v > best)) {
                best = v;
                bi = i;
            }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float v = __shfl_xor_sync(0xffffffffu, best, o);
            const int i = __shfl_xor_sync(0xffffffffu, bi, o);
            if (i != INT_MAX && (bi == INT_MAX || v > best || (v == best && i < bi))) {
                best = v;
                bi = i;
            }
        }
        last = best;
        last_i = bi;
        if (s == 0) first = best;
        if (lane == 0) {
            idx[s] = bi;
            wgt[s] = expf(best - first);
        }
    }
    __syncwarp();
    float sum = 0.f;
    for (int s = 0; s < top; s++) sum += wgt[s];
    __syncwarp();
    for (int s = lane; s < top; s += 32) wgt[s] = wgt[s] / sum;
    __syncwarp();
}

}  // namespace tllm
