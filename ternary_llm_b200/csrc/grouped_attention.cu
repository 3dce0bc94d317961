// Grouped-query attention with per-head norms, rotation and an optional chunk mask (mixers.cuh).
//
// Keys and values live in a ring of cache rows per slot: a chunk mask needs no more rows than a
// chunk and one pass of tokens, whatever the length of the sequence.
//
//   prep   -- norms and rotations of a step's rows (queries in place), keys and values into the cache
//   span   -- one query row against a range of positions, all heads of a key/value head together;
//             decode and short portions (positions split over CTAs, merged afterwards; a single
//             token's norms, rotation and cache append happen in the same launch) and the exact
//             32-bit mode
//   prompt -- BF16, only the tiles some query sees; scores FP32, softmax weights enter the second
//             product as two BF16 numbers.  Long portions of the usual head sizes on tcgen05
//             (grouped_prompt.cu), the rest here: 64 queries of a head per CTA on mma.sync.
#include "grouped_span.cuh"
#include "launch.cuh"
#include "mixers.cuh"
#include "mma_sync.cuh"

namespace tllm {

namespace {

// ---------------------------------------------------------------------------
// Norms, rotations, cache append
// ---------------------------------------------------------------------------
constexpr int kPrepThreads = 256;

// A row is the work of `warps` warps: `hpw` heads each (queries, then keys), then the values.
template <typename T>
__global__ void __launch_bounds__(kPrepThreads)
grouped_prep_kernel(const GroupedArgs<T> a, int warps, int hpw)
{
    pdl_launch_dependents();
    const int unit = (blockIdx.x * kPrepThreads + threadIdx.x) >> 5, lane = threadIdx.x & 31;      // warp of all
    const int row = unit / warps, it = unit - row * warps, b = row / a.g.seq_len, t = row - b * a.g.seq_len;
    pdl_wait();
    const int pos = (a.g.pos_dev ? *a.g.pos_dev : a.g.start_pos) + t;
    if (row >= a.g.n_seq * a.g.seq_len || pos >= a.max_seq) return;
    const int r = pos % a.cache_rows;
    T* proj = a.proj + (size_t)row * a.ld;
    T* kc = a.kc + (size_t)(a.g.first_slot + b) * a.k_slot + (size_t)r * a.kv_heads * a.dim;
    T* vc = a.vc + (size_t)(a.g.first_slot + b) * a.v_slot + (size_t)r * a.kv_heads * a.vdim;
    constexpr int V = Vec16<T>::n;
    const int heads = a.heads + a.kv_heads, head_warps = (heads + hpw - 1) / hpw;
    if (it >= head_warps) {                             // values: 32 pieces of 16 bytes
        const int i = (it - head_warps) * 32 + lane;
        if (i < a.kv_heads * a.vdim / V) reinterpret_cast<uint4*>(vc)[i] = reinterpret_cast<const uint4*>(proj + a.v_off)[i];
        return;
    }
    // in place: an entry is written only by lanes that have read it (the sum of squares comes first)
    const int lanes = 32 / hpw, hh = it * hpw + lane / lanes, h = min(hh, heads - 1);
    const bool q = h < a.heads;
    const T* src = q ? proj + a.q_off + (size_t)h * a.dim : proj + a.k_off + (size_t)(h - a.heads) * a.dim;
    T* dst = q ? const_cast<T*>(src) : kc + (size_t)(h - a.heads) * a.dim;
    if (rotates8(a))
        norm_rotate8<T>(src, a, q ? a.q_norm : a.k_norm, pos, lanes, lane & (lanes - 1), [&](int i, const float (&v)[8]) { if (hh == h) store8(dst + i, v); });
    else
        norm_rotate<T>(src, a, q ? a.q_norm : a.k_norm, pos, [&](int i, float v) { dst[i] = from_f<T>(v); });
}

// ---------------------------------------------------------------------------
// Prompts
// ---------------------------------------------------------------------------
constexpr int kPqWarps = 4, kPqThreads = kPqWarps * 32, kPq = 16 * kPqWarps, kPk = 64;

template <int NV>      // 8-wide output column tiles, even
__global__ void __launch_bounds__(kPqThreads)
grouped_prompt_kernel(const GroupedArgs<bf16> a)
{
    extern __shared__ __align__(16) uint8_t smem_raw[];
    const int D = a.dim, E = a.vdim;
    const int ldq = ((D + 15) & ~15) + 8, ksteps = (D + 15) / 16, ldv = ((E + 15) & ~15) + 8, nv = (E + 15) / 16 * 2;
    bf16* qs = reinterpret_cast<bf16*>(smem_raw);               // [64][ldq]
    bf16* ks = qs + kPq * ldq;                                  // [2][64][ldq]
    bf16* vs = ks + 2 * kPk * ldq;                              // [2][64][ldv]
    pdl_launch_dependents();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, tq = lane & 3;
    const int h = blockIdx.y, g = h / (a.heads / a.kv_heads), b = blockIdx.z, n = a.g.seq_len;
    const int q0 = (gridDim.x - 1 - blockIdx.x) * kPq, nq = min(kPq, n - q0);
    pdl_wait();
    const int pos0 = (a.g.pos_dev ? *a.g.pos_dev : a.g.start_pos) + q0;       // position of the tile's first query
    const int hi = pos0 + nq;                                                 // positions [lo, hi) are seen by some query
    const int lo = first_seen(pos0, a.chunk), lo_last = first_seen(hi - 1, a.chunk);
    const bf16* kc = a.kc + (size_t)(a.g.first_slot + b) * a.k_slot + (size_t)g * D;
    const bf16* vc = a.vc + (size_t)(a.g.first_slot + b) * a.v_slot + (size_t)g * E;
    const size_t krow = (size_t)a.kv_heads * D, vrow = (size_t)a.kv_heads * E;
    const int pk = (ldq - 8) / 8, pv = (ldv - 8) / 8;                         // 16-byte pieces of a row, zero behind D and E
    const uint32_t mk = 0xffffffffu / pk + 1, mv = 0xffffffffu / pv + 1;      // i / pieces as a multiplication
    for (int i = tid; i < kPq * pk; i += kPqThreads) {
        const int r = i / pk, c = (i - r * pk) * 8;
        const bool v = r < nq && c < D;
        cp16(qs + r * ldq + c, v ? a.proj + (size_t)(b * n + q0 + r) * a.ld + a.q_off + (size_t)h * D + c : a.proj, v);
    }
    auto load_tile = [&](int k0, int stage) {
        bf16 *kd = ks + (size_t)stage * kPk * ldq, *vd = vs + (size_t)stage * kPk * ldv;
        const int base = k0 % a.cache_rows;
        for (int i = tid; i < kPk * pk; i += kPqThreads) {
            const int r = pk == 1 ? i : (int)__umulhi((uint32_t)i, mk), c = (i - r * pk) * 8;
            const int ring = base + r < a.cache_rows ? base + r : base + r - a.cache_rows;
            const bool v = k0 + r < hi && c < D;
            cp16(kd + r * ldq + c, v ? kc + (size_t)ring * krow + c : kc, v);
        }
        for (int i = tid; i < kPk * pv; i += kPqThreads) {
            const int r = pv == 1 ? i : (int)__umulhi((uint32_t)i, mv), c = (i - r * pv) * 8;
            const int ring = base + r < a.cache_rows ? base + r : base + r - a.cache_rows;
            const bool v = k0 + r < hi && c < E;
            cp16(vd + r * ldv + c, v ? vc + (size_t)ring * vrow + c : vc, v);
        }
        cp_commit();
    };
    float o[NV][4];
#pragma unroll
    for (int j = 0; j < NV; j++)
#pragma unroll
        for (int e = 0; e < 4; e++) o[j][e] = 0.f;
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
    const float scale2 = a.scale * kLog2e;
    const int row = warp * 16 + gq;                            // rows row and row + 8 of the tile
    const int from[2] = {first_seen(pos0 + row, a.chunk), first_seen(pos0 + row + 8, a.chunk)};
    load_tile(lo, 0);
    int stage = 0;
    for (int k0 = lo; k0 < hi; k0 += kPk, stage ^= 1) {
        if (k0 + kPk < hi) {
            load_tile(k0 + kPk, stage ^ 1);
            cp_wait<1>();
        } else {
            cp_wait<0>();
        }
        __syncthreads();
        const bf16 *kt = ks + (size_t)stage * kPk * ldq, *vt = vs + (size_t)stage * kPk * ldv;
        float s[8][4];
#pragma unroll
        for (int j = 0; j < 8; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) s[j][e] = 0.f;
#pragma unroll 2
        for (int k = 0; k < ksteps; k++) {
            uint32_t fa[4];
            ldsm4(fa, qs + (warp * 16 + (lane & 15)) * ldq + k * 16 + (lane >> 4) * 8);
#pragma unroll
            for (int j = 0; j < 8; j += 2) {                   // 16 positions per load
                uint32_t fb[4];
                ldsm4(fb, kt + (j * 8 + (lane & 7) + (lane >> 4) * 8) * ldq + k * 16 + ((lane >> 3) & 1) * 8);
                mma16816(s[j], fa, fb[0], fb[1]);
                mma16816(s[j + 1], fa, fb[2], fb[3]);
            }
        }
        const bool edge = k0 + kPk > pos0 + 1 || k0 < lo_last;  // some (query, position) pair of the tile is masked
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int j = 0; j < 8; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                float v = s[j][e] * scale2;
                const int p = k0 + j * 8 + 2 * tq + (e & 1);
                if (edge && (p > pos0 + row + (e >> 1) * 8 || p < from[e >> 1])) v = -INFINITY;
                s[j][e] = v;
                mx[e >> 1] = fmaxf(mx[e >> 1], v);
            }
        float cr[2], m_ref[2];
#pragma unroll
        for (int e = 0; e < 2; e++) {
            mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 1));
            mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 2));
            const float m_new = fmaxf(m_run[e], mx[e]);
            m_ref[e] = m_new == -INFINITY ? 0.f : m_new;       // nothing of the row's chunk so far
            cr[e] = exp2_neg(m_run[e] - m_ref[e]);
            m_run[e] = m_new;
            l_run[e] *= cr[e];
        }
        if (__any_sync(0xffffffffu, cr[0] != 1.f || cr[1] != 1.f)) {
#pragma unroll
            for (int j = 0; j < NV; j++) {
                o[j][0] *= cr[0];
                o[j][1] *= cr[0];
                o[j][2] *= cr[1];
                o[j][3] *= cr[1];
            }
        }
#pragma unroll
        for (int k = 0; k < 4; k++) {                          // 16 positions per step
            uint32_t fh[4], fl[4];
#pragma unroll
            for (int q = 0; q < 2; q++) {
                float (&v)[4] = s[2 * k + q];
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    v[e] = exp2_neg(v[e] - m_ref[e >> 1]);
                    l_run[e >> 1] += v[e];
                }
                split2(v[0], v[1], fh[2 * q], fl[2 * q]);
                split2(v[2], v[3], fh[2 * q + 1], fl[2 * q + 1]);
            }
#pragma unroll
            for (int j = 0; j < NV; j += 2) {
                if (j < nv) {
                    uint32_t fb[4];
                    ldsm4t(fb, vt + (k * 16 + (lane & 15)) * ldv + j * 8 + (lane >> 4) * 8);
                    mma16816(o[j], fh, fb[0], fb[1]);
                    mma16816(o[j + 1], fh, fb[2], fb[3]);
                    mma16816(o[j], fl, fb[0], fb[1]);
                    mma16816(o[j + 1], fl, fb[2], fb[3]);
                }
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int e = 0; e < 2; e++) {
        float l = l_run[e];
        l += __shfl_xor_sync(0xffffffffu, l, 1);
        l += __shfl_xor_sync(0xffffffffu, l, 2);
        const int r = row + e * 8;
        if (r >= nq) continue;
        const float f = a.out_scale / l;
        bf16* op = a.out + (size_t)(b * n + q0 + r) * a.ld_out + (size_t)h * E;
#pragma unroll
        for (int j = 0; j < NV; j++) {
            const int c = j * 8 + 2 * tq;
            if (c < E) *reinterpret_cast<__nv_bfloat162*>(op + c) = __floats2bfloat162_rn(o[j][2 * e] * f, o[j][2 * e + 1] * f);
        }
    }
}

constexpr int kPromptFrom = 16;       // tokens from which the tensor-core kernel runs

size_t prompt_smem(int dim, int vdim)
{
    const size_t ldq = ((size_t)(dim + 15) / 16) * 16 + 8, ldv = ((size_t)(vdim + 15) / 16) * 16 + 8;
    return ((kPq + 2 * kPk) * ldq + 2 * kPk * ldv) * sizeof(bf16);
}

template <typename T, int TK, bool ONE>
__global__ void __launch_bounds__(kSpanThreads)
grouped_span_kernel(const GroupedArgs<T> a, float* __restrict__ ws, int hb, int blocks)
{
    extern __shared__ __align__(16) uint8_t smem_raw[];
    pdl_launch_dependents();
    pdl_wait();
    grouped_span<T, TK, ONE>(a, ws, hb, blocks, smem_raw, blockIdx.x, blockIdx.y, blockIdx.z, gridDim.z);
}

constexpr int kMergeThreads = 128;

template <typename T, int TK>
__global__ void __launch_bounds__(kMergeThreads)
grouped_merge_kernel(const GroupedArgs<T> a, const float* __restrict__ ws, int nsplit)
{
    __shared__ float wgt[kSpanMaxSplit];
    pdl_launch_dependents();
    pdl_wait();
    grouped_merge<T, TK>(a, ws, nsplit, blockIdx.x, blockIdx.y, wgt);
}

template <typename T, int TK, bool ONE>
int span_tk(const GroupedArgs<T>& a, float* ws, const SpanPlan& p, cudaStream_t stream)
{
    const auto kernel = grouped_span_kernel<T, TK, ONE>;
    if (p.smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)p.smem);
    const int st = launch_pdl("grouped_span", kernel, dim3(a.g.rows(), a.kv_heads * p.blocks, p.nsplit), dim3(kSpanThreads), p.smem, stream, a, ws,
                              p.hb, p.blocks);
    if (st || p.nsplit == 1) return st;
    return launch_pdl("grouped_merge", grouped_merge_kernel<T, TK>, dim3(a.g.rows(), a.heads), dim3(kMergeThreads), 0, stream, a, ws, p.nsplit);
}

template <typename T>
int span_path(const GroupedArgs<T>& a, float* ws, cudaStream_t stream)
{
    const SpanPlan p = span_plan(a.g.rows(), a.heads, a.kv_heads, a.dim, a.vdim, a.max_seq, a.chunk, sizeof(T));
    if (p.nsplit > 1 && !ws) return fail(TLLM_ERR_NULL, "grouped attention: no workspace");
    if (a.g.seq_len == 1) return p.tk == 64 ? span_tk<T, 64, true>(a, ws, p, stream) : span_tk<T, 16, true>(a, ws, p, stream);
    return p.tk == 64 ? span_tk<T, 64, false>(a, ws, p, stream) : span_tk<T, 16, false>(a, ws, p, stream);
}

bool prompt_fits(const GroupedArgs<float>&) { return false; }
bool prompt_fits(const GroupedArgs<bf16>& a) { return a.g.seq_len >= kPromptFrom && a.vdim <= 256 && prompt_smem(a.dim, a.vdim) <= kSmemLimit; }
int prompt_path(const GroupedArgs<float>&, cudaStream_t) { return TLLM_ERR_SHAPE; }
int prompt_path(const GroupedArgs<bf16>& a, cudaStream_t stream)
{
    if (grouped_prompt_tcgen05_supported(a)) return launch_grouped_prompt_tcgen05(a, stream);
    const dim3 grid((a.g.seq_len + kPq - 1) / kPq, a.heads, a.g.n_seq), block(kPqThreads);
    const size_t smem = prompt_smem(a.dim, a.vdim);
    const int nv = (a.vdim + 15) / 16 * 2;
#define TLLM_CASE(N)                                                                                                             \
    if (nv <= N) {                                                                                                                \
        if (smem > 48 * 1024) cudaFuncSetAttribute(grouped_prompt_kernel<N>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        return launch_pdl("grouped_prompt", grouped_prompt_kernel<N>, grid, block, smem, stream, a);                              \
    }
    TLLM_CASE(4)
    TLLM_CASE(8)
    TLLM_CASE(16)
    TLLM_CASE(32)
#undef TLLM_CASE
    return fail(TLLM_ERR_SHAPE, "grouped attention: vdim=%d", a.vdim);
}

}  // namespace

int grouped_cache_rows(int max_seq, int chunk, int rows)
{
    const long long need = ((long long)chunk + rows + 127) / 128 * 128;       // whole tiles of the prompt kernel
    return chunk > 0 && need < max_seq ? (int)need : max_seq;
}

bool grouped_supported(int heads, int kv_heads, int dim, int vdim)
{
    return heads >= 1 && kv_heads >= 1 && heads % kv_heads == 0 && dim >= 8 && dim % 8 == 0 && vdim >= 8 && vdim % 8 == 0 &&
           vdim <= kSpanAcc * 2 * kSpanThreads && span_smem(1, dim, vdim, 16, 4) <= kSmemLimit / 2;
}

size_t grouped_workspace_floats(int heads, int vdim)
{
    // split steps have at most kSpanTargetCtas CTAs of up to kSpanHeads heads each
    const size_t recs = (size_t)kSpanTargetCtas * (heads < kSpanHeads ? heads : kSpanHeads);
    return recs * (vdim + 2);
}

template <typename T>
int launch_grouped_attention(const GroupedArgs<T>& a, float* ws, cudaStream_t stream)
{
    if (a.g.rows() == 0) return TLLM_OK;
    const int bad = check_grouped(a);
    if (bad) return bad;
    if (a.g.seq_len > 1) {
        if (a.cache_rows < a.max_seq && (a.chunk < 1 || a.chunk + a.g.seq_len > a.cache_rows))
            return fail(TLLM_ERR_SHAPE, "grouped attention: %d tokens with %d cache rows", a.g.seq_len, a.cache_rows);
        const int hpw = !rotates8(a) || a.dim > 128 ? 1 : a.dim > 64 ? 2 : 4, piece = 32 * Vec16<T>::n;
        const int warps = (a.heads + a.kv_heads + hpw - 1) / hpw + (a.kv_heads * a.vdim + piece - 1) / piece;
        const unsigned ctas = ((unsigned)a.g.rows() * warps + kPrepThreads / 32 - 1) / (kPrepThreads / 32);
        const int st = launch_pdl("grouped_prep", grouped_prep_kernel<T>, dim3(ctas), dim3(kPrepThreads), 0, stream, a, warps, hpw);
        if (st) return st;
        if (prompt_fits(a)) return prompt_path(a, stream);
    }
    return span_path<T>(a, ws, stream);
}
template int launch_grouped_attention<bf16>(const GroupedArgs<bf16>&, float*, cudaStream_t);
template int launch_grouped_attention<float>(const GroupedArgs<float>&, float*, cudaStream_t);

}  // namespace tllm
