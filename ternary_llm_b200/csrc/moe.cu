// Mixture of experts: choice of a token's experts, products with few rows, and the gathering of
// many rows into groups of one expert each.
//
// Few rows (decode): a token's chosen experts are streamed from memory once per token by the dense
// GEMV (LinearArgs::route).  Every CTA makes the choice itself from the router's logits, so there
// is no launch in between; the down projection sums over the chosen experts inside a row.
// Many rows (prompts): one launch chooses and counts, the next gathers the rows of each expert
// into groups of 128 and writes the table of groups, and the dense GEMM runs over the groups that
// exist (LinearArgs::group).  The weighted sum over a token's experts is part of the residual
// chain (NormArgs::parts).  A row's result does not depend on its place in a group.
#include "launch.cuh"
#include "mixers.cuh"
#include "route.cuh"

namespace tllm {

namespace {

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
    choose_experts(a.z + (size_t)row * a.ld_z, a.experts, a.top, idx, wgt);
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
            for (int g = first[e]; g < first[e + 1]; g++) {
                a.group[3 * g] = e;
                a.group[3 * g + 1] = first[e];
                a.group[3 * g + 2] = first[e + 1] - first[e];
            }
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

template <typename T>
int check_experts(const ExpertArgs<T>& a)
{
    if (a.experts < 1 || a.top < 1 || a.top > a.experts || a.w % 8 || a.ff % 8 || a.ff < 8 || a.ld_z < a.experts)
        return fail(TLLM_ERR_SHAPE, "experts: %d of %d, width=%d ff=%d", a.top, a.experts, a.w, a.ff);
    return TLLM_OK;
}

}  // namespace

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
    if (st) return st;
    LinearArgs<T> l;
    l.route.z = a.z;
    l.route.ld_z = a.ld_z;
    l.route.experts = a.experts;
    l.route.top = a.top;
    l.w = a.gate_up;
    l.ldw = l.K = l.ldx = a.w;
    l.w_rows = 2 * a.ff;
    l.x = a.h;
    l.y = a.hidden;
    l.ldy = l.N = a.ff;
    l.M = a.rows;
    l.act = a.act;
    l.glu = true;
    if ((st = launch_dense_gemv_routed<T>(l, false, stream))) return st;
    LinearArgs<T> d;
    d.route = l.route;
    d.w = a.down;
    d.ldw = d.K = a.ff;
    d.w_rows = d.N = d.ldy = a.w;
    d.x = a.hidden;
    d.ldx = a.ff * a.top;
    d.y = a.y;
    d.y_f32 = true;
    d.M = a.rows;
    return launch_dense_gemv_routed<T>(d, true, stream);
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
