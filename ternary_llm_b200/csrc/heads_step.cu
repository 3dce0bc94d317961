// A decode step of attention and linear attention side by side: the two read the same projection
// and neither waits for the other, so their CTAs share a launch, and so do the merge of the
// attention's ranges and the norm of the other's output.
#include "grouped_span.cuh"
#include "matrix_step.cuh"

namespace tllm {

namespace {

static_assert(kSpanThreads == kSeqThreads && kSpanThreads == kGnThreads, "one block size");

template <typename T, int TK>
__global__ void __launch_bounds__(kSpanThreads)
heads_step_kernel(const GroupedArgs<T> a, const MatrixScanArgs<T> m, float* __restrict__ ws, int hb, int blocks, int nsplit, int log_lpc, int col_blocks)
{
    extern __shared__ __align__(16) uint8_t smem[];
    pdl_launch_dependents();
    pdl_wait();
    const int seq_ctas = col_blocks * m.heads * m.g.n_seq;
    int i = blockIdx.x;
    if (i < seq_ctas) {
        const int bx = i % col_blocks, h = i / col_blocks % m.heads, b = i / (col_blocks * m.heads);
        matrix_one<T, false, false>(m, GatedNormArgs<T>(), log_lpc, nullptr, bx, h, b);
        return;
    }
    i -= seq_ctas;
    const int per_row = a.kv_heads * blocks * nsplit, row = i / per_row;
    i -= row * per_row;
    grouped_span<T, TK, true>(a, ws, hb, blocks, smem, row, i / nsplit, i % nsplit, nsplit);
}

template <typename T, int TK>
__global__ void __launch_bounds__(kGnThreads)
heads_finish_kernel(const GroupedArgs<T> a, const GatedNormArgs<T> norm, const float* __restrict__ ws, int nsplit)
{
    __shared__ float sh[kSpanMaxSplit];
    pdl_launch_dependents();
    pdl_wait();
    const int i = blockIdx.x;
    if (i < norm.rows) {
        gated_norm_row<T>(norm, i, sh);
        return;
    }
    const int j = i - norm.rows;
    grouped_merge<T, TK>(a, ws, nsplit, j / a.heads, j % a.heads, sh);
}

template <typename T, int TK>
int step_tk(const GroupedArgs<T>& a, const MatrixScanArgs<T>& m, const GatedNormArgs<T>& norm, float* ws, const SpanPlan& p, cudaStream_t stream)
{
    const SeqPlan q = seq_plan(m.dim, m.vdim);
    const size_t smem = p.smem;
    const int rows = a.g.n_seq, ctas = q.blocks * m.heads * rows + rows * a.kv_heads * p.blocks * p.nsplit;
    const auto kernel = heads_step_kernel<T, TK>;
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    const int st = launch_pdl("heads_step", kernel, dim3(ctas), dim3(kSpanThreads), smem, stream, a, m, ws, p.hb, p.blocks, p.nsplit, q.log_lpc, q.blocks);
    if (st) return st;
    return launch_pdl("heads_finish", heads_finish_kernel<T, TK>, dim3(norm.rows + (p.nsplit > 1 ? rows * a.heads : 0)), dim3(kGnThreads), 0, stream, a,
                      norm, ws, p.nsplit);
}

}  // namespace

template <typename T>
int launch_heads_step(const GroupedArgs<T>& a, const MatrixScanArgs<T>& m, const GatedNormArgs<T>& norm, float* ws, cudaStream_t stream)
{
    if (a.g.n_seq == 0) return TLLM_OK;
    int st = check_grouped(a);
    if (!st) st = check_matrix_scan(m);
    if (st) return st;
    if (a.g.seq_len != 1 || m.g.seq_len != 1 || m.g.n_seq != a.g.n_seq || m.delta || !ws)
        return fail(TLLM_ERR_SHAPE, "heads_step: %d tokens of %d sequences", a.g.seq_len, a.g.n_seq);
    const SpanPlan p = span_plan(a.g.rows(), a.heads, a.kv_heads, a.dim, a.vdim, a.max_seq, a.chunk, sizeof(T));
    return p.tk == 64 ? step_tk<T, 64>(a, m, norm, ws, p, stream) : step_tk<T, 16>(a, m, norm, ws, p, stream);
}
template int launch_heads_step<bf16>(const GroupedArgs<bf16>&, const MatrixScanArgs<bf16>&, const GatedNormArgs<bf16>&, float*, cudaStream_t);
template int launch_heads_step<float>(const GroupedArgs<float>&, const MatrixScanArgs<float>&, const GatedNormArgs<float>&, float*, cudaStream_t);

}  // namespace tllm
