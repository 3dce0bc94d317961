// Mixture of experts: choice of a token's experts, products with few rows, and the gathering of
// many rows into groups of one expert each.
//
// Few rows (decode): a token's chosen experts are streamed from memory once per token.  Every CTA
// makes the choice itself from the router's logits, so there is no launch in between; the down
// projection sums over the chosen experts inside the row's dot product.
// Many rows (prompts): one launch chooses and counts, the next gathers the rows of each expert
// into groups of 128 and writes the table of groups, and the dense GEMM runs over the groups that
// exist (LinearArgs::group).  The weighted sum over a token's experts is part of the residual
// chain (NormArgs::parts).  A row's result does not depend on its place in a group.
#include <cfloat>

#include "launch.cuh"
#include "mixers.cuh"

namespace tllm {

namespace {

// One warp: the `top` largest of z[0..experts) in order and the softmax over them; idx, wgt in
// shared memory.  Lane l looks at entries l, l + 32, ...
__device__ __forceinline__ void choose(const float* z, int experts, int top, int* idx, float* wgt)
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

// ---------------------------------------------------------------------------
// Few rows
// ---------------------------------------------------------------------------
constexpr int kFewWarps = 8, kPieces = 8;       // 16-byte pieces a lane requests together

// sum over a row of nv pieces against a vector in shared memory
template <typename T>
__device__ __forceinline__ void dot_pieces(const T* row, const T* xs, int nv, float& acc)
{
    constexpr int V = Vec16<T>::n;
    const int lane = threadIdx.x & 31;
    for (int c0 = lane; c0 - lane < nv; c0 += 32 * kPieces) {
        uint4 w[kPieces];
#pragma unroll
        for (int u = 0; u < kPieces; u++) {
            const int c = c0 + u * 32;
            w[u] = c < nv ? __ldcs(reinterpret_cast<const uint4*>(row) + c) : make_uint4(0, 0, 0, 0);
        }
#pragma unroll
        for (int u = 0; u < kPieces; u++) {
            const int c = min(c0 + u * 32, nv - 1);
            float wf[V], xf[V];
            Vec16<T>::unpack(w[u], wf);
            Vec16<T>::unpack(reinterpret_cast<const uint4*>(xs)[c], xf);
#pragma unroll
            for (int j = 0; j < V; j++) acc = fmaf(wf[j], xf[j], acc);
        }
    }
}

// DOWN = false: hidden[row, s] = act(gate h) * (up h) of the row's s-th expert (grid.y = row * top + s)
// DOWN = true:  y[row] = sum_s weight_s * down_s hidden[row, s]                (grid.y = row)
template <typename T, bool DOWN>
__global__ void __launch_bounds__(kFewWarps * 32)
experts_few_kernel(const ExpertArgs<T> a)
{
    extern __shared__ __align__(16) uint8_t smem[];
    const int K = DOWN ? a.ff : a.w, parts = DOWN ? a.top : 1, nv = K / Vec16<T>::n;
    T* xs = reinterpret_cast<T*>(smem);                          // [parts][K]
    float* wgt = reinterpret_cast<float*>(xs + (size_t)parts * K);
    int* idx = reinterpret_cast<int*>(wgt + a.top);
    pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int row = DOWN ? blockIdx.y : blockIdx.y / a.top, slot = DOWN ? 0 : blockIdx.y - row * a.top;
    pdl_wait();
    if (warp == 0) choose(a.z + (size_t)row * a.ld_z, a.experts, a.top, idx, wgt);
    const uint4* src = reinterpret_cast<const uint4*>(DOWN ? a.hidden + (size_t)row * a.top * K : a.h + (size_t)row * K);
    for (int i = threadIdx.x; i < parts * nv; i += kFewWarps * 32) reinterpret_cast<uint4*>(xs)[i] = src[i];
    __syncthreads();
    const int N = DOWN ? a.w : a.ff;
    for (int n = blockIdx.x * kFewWarps + warp; n < N; n += gridDim.x * kFewWarps) {
        if (DOWN) {
            float y = 0.f;
            for (int s = 0; s < parts; s++) {
                float acc = 0.f;
                dot_pieces<T>(a.down + ((size_t)idx[s] * a.w + n) * K, xs + (size_t)s * K, nv, acc);
                y = fmaf(wgt[s], acc, y);
            }
            y = warp_sum(y);
            if (lane == 0) a.y[(size_t)row * a.w + n] = y;
        } else {
            const T* g = a.gate_up + ((size_t)idx[slot] * 2 * a.ff + n) * K;
            float gate = 0.f, up = 0.f;
            dot_pieces<T>(g, xs, nv, gate);
            dot_pieces<T>(g + (size_t)a.ff * K, xs, nv, up);
            gate = warp_sum(gate);
            up = warp_sum(up);
            if (lane == 0) a.hidden[((size_t)row * a.top + slot) * a.ff + n] = from_f<T>(apply_act(a.act, gate) * up);
        }
    }
}

// ---------------------------------------------------------------------------
// Many rows
// ---------------------------------------------------------------------------
constexpr int kChooseWarps = 8;

template <typename T>
__global__ void __launch_bounds__(kChooseWarps * 32)
experts_choose_kernel(const ExpertArgs<T> a)
{
    extern __shared__ __align__(16) uint8_t smem[];
    float* wgt = reinterpret_cast<float*>(smem);
    int* idx = reinterpret_cast<int*>(wgt + kChooseWarps * a.top);
    pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row = blockIdx.x * kChooseWarps + warp;
    pdl_wait();
    if (row >= a.rows) return;
    wgt += warp * a.top;
    idx += warp * a.top;
    choose(a.z + (size_t)row * a.ld_z, a.experts, a.top, idx, wgt);
    for (int s = lane; s < a.top; s += 32) {
        a.chosen[(size_t)row * a.top + s] = idx[s];
        a.part_w[(size_t)row * a.top + s] = wgt[s];
        atomicAdd(a.counts + idx[s], 1);
    }
}

constexpr int kGatherThreads = 128;

// One CTA per row: its place in each chosen expert's group, and the copy.  counts: tokens per
// expert, then places given out per expert.
template <typename T>
__global__ void __launch_bounds__(kGatherThreads)
experts_gather_kernel(const ExpertArgs<T> a)
{
    extern __shared__ __align__(16) uint8_t smem[];
    int* first = reinterpret_cast<int*>(smem);          // [experts + 1], in groups
    int* place = first + a.experts + 1;                 // [top]
    pdl_launch_dependents();
    const int row = blockIdx.x, tid = threadIdx.x;
    pdl_wait();
    if (tid < 32) {                                     // exclusive sums of the groups per expert
        int base = 0;
        for (int e0 = 0; e0 < a.experts; e0 += 32) {
            const int e = e0 + tid, n = e < a.experts ? (a.counts[e] + kGroupRows - 1) / kGroupRows : 0;
            int s = n;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int v = __shfl_up_sync(0xffffffffu, s, o);
                if (tid >= o) s += v;
            }
            if (e < a.experts) first[e] = base + s - n;
            base += __shfl_sync(0xffffffffu, s, 31);
        }
        if (tid == 0) first[a.experts] = base;
    }
    __syncthreads();
    if (row == 0) {
        for (int e = tid; e < a.experts; e += kGatherThreads)
            for (int g = first[e]; g < first[e + 1]; g++) a.group[g] = e;
        if (tid == 0) *a.groups = first[a.experts];
    }
    for (int s = tid; s < a.top; s += kGatherThreads) {
        const int e = a.chosen[(size_t)row * a.top + s];
        const int p = first[e] * kGroupRows + atomicAdd(a.counts + a.experts + e, 1);
        place[s] = p;
        a.part_row[(size_t)row * a.top + s] = p;
    }
    __syncthreads();
    const int nv = a.w / Vec16<T>::n;
    const uint4* src = reinterpret_cast<const uint4*>(a.h + (size_t)row * a.w);
    for (int i = tid; i < nv; i += kGatherThreads) {
        const uint4 v = src[i];
        for (int s = 0; s < a.top; s++) reinterpret_cast<uint4*>(a.gathered + (size_t)place[s] * a.w)[i] = v;
    }
}

constexpr size_t kSmemLimit = 220 * 1024;

template <typename T>
int check_experts(const ExpertArgs<T>& a)
{
    if (a.experts < 1 || a.top < 1 || a.top > a.experts || a.w % 8 || a.ff % 8 || a.ff < 8 || a.ld_z < a.experts)
        return fail(TLLM_ERR_SHAPE, "experts: %d of %d, width=%d ff=%d", a.top, a.experts, a.w, a.ff);
    return TLLM_OK;
}

size_t few_smem(int top, int ff, int w, size_t es, bool down) { return (down ? (size_t)top * ff : (size_t)w) * es + (size_t)top * 8; }

template <typename T, bool DOWN>
int few(const ExpertArgs<T>& a, cudaStream_t stream)
{
    const size_t smem = few_smem(a.top, a.ff, a.w, sizeof(T), DOWN);
    if (smem > kSmemLimit) return fail(TLLM_ERR_SHAPE, "experts: %d of %d, ff=%d do not fit shared memory", a.top, a.experts, a.ff);
    if (smem > 48 * 1024) cudaFuncSetAttribute(experts_few_kernel<T, DOWN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    const int ny = DOWN ? a.rows : a.rows * a.top, n = DOWN ? a.w : a.ff;
    int gx = (n + kFewWarps - 1) / kFewWarps;
    const int cap = (6 * 148 + ny - 1) / ny;
    if (gx > cap) gx = cap;
    return launch_pdl("experts", experts_few_kernel<T, DOWN>, dim3(gx, ny), dim3(kFewWarps * 32), smem, stream, a);
}

}  // namespace

bool experts_few_fits(int top, int ff, int w, size_t element)
{
    return few_smem(top, ff, w, element, true) <= kSmemLimit && few_smem(top, ff, w, element, false) <= kSmemLimit;
}

int expert_rows(int rows, int top, int experts)
{
    // every expert in use wastes less than one group
    const long long used = (long long)rows * top < experts ? (long long)rows * top : experts;
    return (int)(((long long)rows * top + used * (kGroupRows - 1)) / kGroupRows * kGroupRows);
}

template <typename T>
int launch_experts_few(const ExpertArgs<T>& a, cudaStream_t stream)
{
    if (a.rows == 0) return TLLM_OK;
    int st = check_experts(a);
    if (!st) st = few<T, false>(a, stream);
    if (!st) st = few<T, true>(a, stream);
    return st;
}

template <typename T>
int launch_experts_gather(const ExpertArgs<T>& a, cudaStream_t stream)
{
    if (a.rows == 0) return TLLM_OK;
    int st = check_experts(a);
    if (st) return st;
    if (cudaMemsetAsync(a.counts, 0, (size_t)2 * a.experts * sizeof(int), stream) != cudaSuccess)
        return fail(TLLM_ERR_LAUNCH, "experts: %s", cudaGetErrorString(cudaGetLastError()));
    const size_t s1 = (size_t)kChooseWarps * a.top * 8, s2 = (size_t)(a.experts + 1 + a.top) * sizeof(int);
    if (s1 > 48 * 1024 || s2 > 48 * 1024) return fail(TLLM_ERR_SHAPE, "experts: %d of %d", a.top, a.experts);
    st = launch_pdl("experts_choose", experts_choose_kernel<T>, dim3((a.rows + kChooseWarps - 1) / kChooseWarps), dim3(kChooseWarps * 32), s1,
                    stream, a);
    if (st) return st;
    return launch_pdl("experts_gather", experts_gather_kernel<T>, dim3(a.rows), dim3(kGatherThreads), s2, stream, a);
}

#define TLLM_INSTANTIATE(T)                                               \
    template int launch_experts_few<T>(const ExpertArgs<T>&, cudaStream_t); \
    template int launch_experts_gather<T>(const ExpertArgs<T>&, cudaStream_t);
TLLM_INSTANTIATE(bf16)
TLLM_INSTANTIATE(float)
#undef TLLM_INSTANTIATE

}  // namespace tllm
