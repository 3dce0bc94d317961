// Grouped-query attention over prompts on the 5th-generation tensor cores (BF16, head sizes 64 and
// 128; the other sizes run on mma.sync, grouped_attention.cu).
//
// A CTA takes 128 queries of one head and walks over tiles of 128 positions that some of its queries
// sees; two CTAs share an SM, so that one's softmax runs beside the other's products.  Roles: a TMA
// producer, one thread that issues tcgen05.mma, four warps with a query row per thread.
//   S = Q K^T      both operands in shared memory, 128 FP32 columns of tensor memory
//   softmax        a thread reads its row; the weights go back over S as two BF16 numbers each
//   O += P V       weights from tensor memory, values as they lie in the cache (feature-major
//                  operand); the high and the low parts are two products
// The running maximum moves only when it grows by more than 2^8: the sums stay far inside FP32, and
// the output in tensor memory is rescaled a few times per row at most.  All mbarrier waits are
// bounded (see dense_gemm.cu).
#include "launch.cuh"
#include "mixers.cuh"
#include "tcgen05.cuh"

namespace tllm {

namespace {

using namespace gemm;

constexpr int kTile = 128, kThreads = 192;
constexpr int kBlock = kTile * 128;                 // bytes of 64 columns of a tile: 128-byte rows
constexpr uint32_t kTmemCols = 256;                 // S and the weights: 128, O: 128
constexpr float kLog2e = 1.4426950408889634f, kSlack = 8.f;

struct PromptArgs {
    bf16* out;
    int ld_out, heads, per_kv, dim, vdim, n, pos0, chunk, cache_rows;
    float scale2, out_scale;
    int* err;
};

__device__ __forceinline__ int chunk_start(int pos, int chunk) { return chunk > 0 ? pos / chunk * chunk : 0; }

__device__ __forceinline__ uint32_t idesc(int n, bool feature_major)
{
    return (1u << 4) | (1u << 7) | (1u << 10) | ((feature_major ? 1u : 0u) << 16) | ((uint32_t)(n >> 3) << 17) | ((uint32_t)(kTile >> 4) << 24);
}
// operand whose rows are the contracted index: blocks of 64 features kBlock apart, groups of 8 rows 1024 bytes apart
__device__ __forceinline__ uint64_t feature_major_desc(uint32_t addr)
{
    return (make_sw128_desc(addr) & ~((uint64_t)0x3fff << 16)) | ((uint64_t)(kBlock >> 4) << 16);
}
__device__ __forceinline__ void mma_ss(uint32_t d, uint64_t a, uint64_t b, uint32_t id, bool acc)
{
    asm volatile(
        "{ .reg .pred p; setp.ne.b32 p, %4, 0;\n"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p; }"
        ::"r"(d), "l"(a), "l"(b), "r"(id), "r"((uint32_t)acc) : "memory");
}
__device__ __forceinline__ void mma_ts(uint32_t d, uint32_t a, uint64_t b, uint32_t id, bool acc)
{
    asm volatile(
        "{ .reg .pred p; setp.ne.b32 p, %4, 0;\n"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p; }"
        ::"r"(d), "r"(a), "l"(b), "r"(id), "r"((uint32_t)acc) : "memory");
}
__device__ __forceinline__ void tmem_st32(uint32_t taddr, const uint32_t (&r)[32])
{
    asm volatile("tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,"
                 "%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31,%32};"
                 ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),
                 "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]),
                 "r"(r[16]), "r"(r[17]), "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]),
                 "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31]) : "memory");
}
__device__ __forceinline__ void wait_ld() { asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ void wait_st() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ void fence_after() { asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory"); }
__device__ __forceinline__ void fence_before() { asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory"); }

enum Bar { kQFull, kKFull, kKEmpty, kVFull, kVEmpty, kSFull, kPReady, kPvDone, kBars };

__global__ void __launch_bounds__(kThreads, 2)
grouped_prompt_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                         const __grid_constant__ CUtensorMap map_v, const PromptArgs a)
{
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    __shared__ __align__(8) uint64_t bars[kBars];
    __shared__ uint32_t tmem_slot;
    __shared__ int abort_flag;
    pdl_launch_dependents();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int h = blockIdx.y, g = h / a.per_kv, q0 = (gridDim.x - 1 - blockIdx.x) * kTile;       // longest first
    const int nq = min(kTile, a.n - q0), first = a.pos0 + q0, hi = first + nq;                    // positions of the queries
    const int lo = chunk_start(first, a.chunk) & ~(kTile - 1), lo_last = chunk_start(hi - 1, a.chunk);
    const int tiles = (hi - lo + kTile - 1) / kTile, nd = a.dim / 64, ne = a.vdim / 64;
    const uint32_t qs = smem_u32(smem), ks = qs + nd * kBlock, vs = ks + nd * kBlock, bar0 = smem_u32(bars);
    auto bar = [&](int i) { return bar0 + 8u * i; };
    volatile int* abortp = &abort_flag;
    int never = 0;

    if (tid == 0) {
        for (int i = 0; i < kBars; i++) mbar_init(bar(i), i == kPReady ? kTile : 1);
        abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == 5) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_slot)), "r"(kTmemCols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    fence_before();
    __syncthreads();
    fence_after();
    const uint32_t tmem = tmem_slot, tmem_o = tmem + kTile;
    pdl_wait();

    if (warp == 4) {
        // ---------------- TMA producer ----------------
        if (lane == 0) {
            int issued = 0;                                     // tiles whose copies were issued: keys, then values
            mbar_expect_tx(bar(kQFull), nd * kBlock);
            for (int j = 0; j < nd; j++) tma_load_2d(qs + j * kBlock, &map_q, h * a.dim + j * 64, q0, bar(kQFull));
            for (int i = 0; i < 2 * tiles; i++, issued++) {
                const int t = i >> 1, row = (lo + t * kTile) % a.cache_rows;
                const bool v = i & 1;
                if (!mbar_wait(bar(v ? kVEmpty : kKEmpty), (t & 1) ^ 1, abortp)) {
                    abort_flag = 1;
                    break;
                }
                const int blocks = v ? ne : nd;
                mbar_expect_tx(bar(v ? kVFull : kKFull), blocks * kBlock);
                for (int j = 0; j < blocks; j++) {
                    if (v) tma_load_2d(vs + j * kBlock, &map_v, g * a.vdim + j * 64, row, bar(kVFull));
                    else tma_load_2d(ks + j * kBlock, &map_k, g * a.dim + j * 64, row, bar(kKFull));
                }
            }
            // after an abort the copies still in flight must land before the shared memory goes away
            if (*abortp) {
                mbar_wait(bar(kQFull), 0, &never);
                if (issued > 0) mbar_wait(bar(kKFull), ((issued - 1) >> 1) & 1, &never);
                if (issued > 1) mbar_wait(bar(kVFull), ((issued - 2) >> 1) & 1, &never);
            }
        }
    } else if (warp == 5) {
        // ---------------- MMA issuer ----------------
        if (lane == 0) {
            const uint32_t id_s = idesc(kTile, false), id_o = idesc(a.vdim, true);
            bool ok = mbar_wait(bar(kQFull), 0, abortp);
            int done = 0;                                       // tiles whose last product was issued
            for (int t = 0; ok && t < tiles; t++) {
                // the weights of the tile before lie where S goes
                ok = (t == 0 || mbar_wait(bar(kPvDone), (t - 1) & 1, abortp)) && mbar_wait(bar(kKFull), t & 1, abortp);
                if (!ok) break;
                fence_after();
                for (int k = 0; k < a.dim / 16; k++) {
                    const uint32_t o = (k >> 2) * kBlock + (k & 3) * 32;
                    mma_ss(tmem, make_sw128_desc(qs + o), make_sw128_desc(ks + o), id_s, k > 0);
                }
                mma_commit(bar(kKEmpty));
                mma_commit(bar(kSFull));
                ok = mbar_wait(bar(kVFull), t & 1, abortp) && mbar_wait(bar(kPReady), t & 1, abortp);
                if (!ok) break;
                fence_after();
                for (int part = 0; part < 2; part++)
                    for (int k = 0; k < kTile / 16; k++)
                        mma_ts(tmem_o, tmem + part * 64 + k * 8, feature_major_desc(vs + k * 2048), id_o, t > 0 || part > 0 || k > 0);
                mma_commit(bar(kVEmpty));
                mma_commit(bar(kPvDone));
                done++;
            }
            if (!ok) {
                abort_flag = 1;
                // what was issued completes before the memory is given up
                mma_commit(bar(kPvDone));
                mbar_wait(bar(kPvDone), done & 1, &never);
            }
        }
    } else if (warp < 4) {
        // ---------------- softmax: a row per thread ----------------
        const uint32_t row_s = tmem + ((uint32_t)(warp * 32) << 16), row_o = row_s + kTile;
        const int pos = first + tid, from = chunk_start(pos, a.chunk);
        float m = -INFINITY, l = 0.f;
        bool ok = true;
        for (int t = 0; t < tiles; t++) {
            const int k0 = lo + t * kTile;
            ok = __all_sync(0xffffffffu, mbar_wait(bar(kSFull), t & 1, abortp));
            if (!ok) break;
            fence_after();
            uint32_t s[4][32];
            __syncwarp();
#pragma unroll
            for (int i = 0; i < 4; i++) tmem_ld32(row_s + i * 32, s[i]);
            wait_ld();
            const bool edge = k0 + kTile > first + 1 || k0 < lo_last;         // some (query, position) pair of the tile is masked
            float mx = -INFINITY;
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 32; j++) {
                    float v = __uint_as_float(s[i][j]) * a.scale2;
                    const int p = k0 + i * 32 + j;
                    if (edge && (p > pos || p < from)) v = -INFINITY;
                    s[i][j] = __float_as_uint(v);
                    mx = fmaxf(mx, v);
                }
            const bool grows = mx > m + kSlack || (m == -INFINITY && mx > m);
            if (__any_sync(0xffffffffu, grows)) {
                const float f = grows ? exp2_neg(m - mx) : 1.f;               // 0 where nothing was seen before
                if (grows) {
                    m = mx;
                    l *= f;
                }
                if (t > 0) {
#pragma unroll 1
                    for (int c = 0; c < a.vdim; c += 32) {
                        uint32_t o[32];
                        tmem_ld32(row_o + c, o);
                        wait_ld();
#pragma unroll
                        for (int j = 0; j < 32; j++) o[j] = __float_as_uint(__uint_as_float(o[j]) * f);
                        tmem_st32(row_o + c, o);
                    }
                }
            }
            const float ref = m == -INFINITY ? 0.f : m;
#pragma unroll
            for (int half = 0; half < 2; half++) {                            // 64 positions: 32 words of high, 32 of low parts
                uint32_t ph[32], pl[32];
#pragma unroll
                for (int j = 0; j < 32; j++) {
                    const float p0 = exp2_neg(__uint_as_float(s[2 * half + (j >> 4)][2 * (j & 15)]) - ref);
                    const float p1 = exp2_neg(__uint_as_float(s[2 * half + (j >> 4)][2 * (j & 15) + 1]) - ref);
                    l += p0 + p1;
                    const __nv_bfloat162 b = __floats2bfloat162_rn(p0, p1);
                    const float2 r = __bfloat1622float2(b);
                    const __nv_bfloat162 c = __floats2bfloat162_rn(p0 - r.x, p1 - r.y);
                    ph[j] = *reinterpret_cast<const uint32_t*>(&b);
                    pl[j] = *reinterpret_cast<const uint32_t*>(&c);
                }
                tmem_st32(row_s + half * 32, ph);
                tmem_st32(row_s + 64 + half * 32, pl);
            }
            if (k0 + kTile > hi) {
                // rows of the cache behind the last query hold anything: their weights are 0, their values become 0
                ok = __all_sync(0xffffffffu, mbar_wait(bar(kVFull), t & 1, abortp));
                if (!ok) break;
                if (k0 + tid >= hi)
                    for (int j = 0; j < ne * 8; j++)
                        *reinterpret_cast<uint4*>(smem + (size_t)(2 * nd + (j >> 3)) * kBlock + tid * 128 + (j & 7) * 16) = make_uint4(0, 0, 0, 0);
                asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            }
            wait_st();
            fence_before();
            mbar_arrive(bar(kPReady));
        }
        if (ok) ok = __all_sync(0xffffffffu, mbar_wait(bar(kPvDone), (tiles - 1) & 1, abortp));
        if (ok) {
            fence_after();
            const float f = a.out_scale / l;
            bf16* op = a.out + (size_t)(q0 + tid) * a.ld_out + (size_t)h * a.vdim;
#pragma unroll 1
            for (int c = 0; c < a.vdim; c += 32) {
                uint32_t o[32];
                tmem_ld32(row_o + c, o);
                wait_ld();
                if (tid < nq) {
#pragma unroll
                    for (int j = 0; j < 4; j++) {
                        __nv_bfloat162 w[4];
#pragma unroll
                        for (int i = 0; i < 4; i++)
                            w[i] = __floats2bfloat162_rn(__uint_as_float(o[8 * j + 2 * i]) * f, __uint_as_float(o[8 * j + 2 * i + 1]) * f);
                        *reinterpret_cast<uint4*>(op + c + 8 * j) = *reinterpret_cast<const uint4*>(w);
                    }
                }
            }
        } else {
            abort_flag = 1;
        }
    }
    fence_before();
    __syncthreads();
    if (abort_flag && tid == 0) atomicExch(a.err, TLLM_ERR_TIMEOUT);
    if (warp == 5) {
        fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kTmemCols) : "memory");
    }
}

size_t smem_bytes(int dim, int vdim) { return (size_t)(2 * (dim / 64) + vdim / 64) * kBlock + 1024; }

int encode(EncodeTiledFn enc, CUtensorMap* map, const bf16* p, int cols, int rows, size_t ld)
{
    const cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
    const cuuint64_t strides[1] = {(cuuint64_t)ld * sizeof(bf16)};
    const cuuint32_t box[2] = {64, (cuuint32_t)kTile};
    const cuuint32_t estr[2] = {1, 1};
    const CUresult r = enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<bf16*>(p), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                           CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) return fail(TLLM_ERR_LAUNCH, "grouped_prompt: cuTensorMapEncodeTiled failed with %d", (int)r);
    return TLLM_OK;
}

}  // namespace

bool grouped_prompt_tcgen05_supported(const GroupedArgs<bf16>& a)
{
    // the tiles of a ring do not wrap when its rows are a multiple of a tile
    return (a.dim == 64 || a.dim == 128) && (a.vdim == 64 || a.vdim == 128) && a.g.n_seq == 1 && !a.g.pos_dev && a.g.seq_len >= kTile &&
           (a.cache_rows >= a.max_seq || a.cache_rows % kTile == 0) && a.ld_out % 8 == 0 &&
           ((reinterpret_cast<uintptr_t>(a.out) | reinterpret_cast<uintptr_t>(a.proj + a.q_off) | reinterpret_cast<uintptr_t>(a.kc) |
             reinterpret_cast<uintptr_t>(a.vc)) & 15) == 0;
}

int launch_grouped_prompt_tcgen05(const GroupedArgs<bf16>& a, cudaStream_t stream)
{
    EncodeTiledFn enc = encode_fn();
    if (!enc) return fail(TLLM_ERR_LAUNCH, "cuTensorMapEncodeTiled is not available from this driver");
    const bf16 *kc = a.kc + (size_t)a.g.first_slot * a.k_slot, *vc = a.vc + (size_t)a.g.first_slot * a.v_slot;
    CUtensorMap mq, mk, mv;
    int st;
    if ((st = encode(enc, &mq, a.proj + a.q_off, a.heads * a.dim, a.g.seq_len, a.ld))) return st;
    if ((st = encode(enc, &mk, kc, a.kv_heads * a.dim, a.cache_rows, (size_t)a.kv_heads * a.dim))) return st;
    if ((st = encode(enc, &mv, vc, a.kv_heads * a.vdim, a.cache_rows, (size_t)a.kv_heads * a.vdim))) return st;
    PromptArgs p;
    p.out = a.out;
    p.ld_out = a.ld_out;
    p.heads = a.heads;
    p.per_kv = a.heads / a.kv_heads;
    p.dim = a.dim;
    p.vdim = a.vdim;
    p.n = a.g.seq_len;
    p.pos0 = a.g.start_pos;
    p.chunk = a.chunk;
    p.cache_rows = a.cache_rows;
    p.scale2 = a.scale * kLog2e;
    p.out_scale = a.out_scale;
    p.err = device_error_flag();
    if (!p.err) return fail(TLLM_ERR_LAUNCH, "device scratch unavailable");
    static bool attr[64] = {};
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev < 0 || dev >= 64) return fail(TLLM_ERR_LAUNCH, "grouped_prompt: no current device");
    if (!attr[dev]) {
        cudaFuncSetAttribute(grouped_prompt_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_bytes(128, 128));
        attr[dev] = true;
    }
    return launch_pdl("grouped_prompt", grouped_prompt_tc_kernel, dim3((a.g.seq_len + kTile - 1) / kTile, a.heads), dim3(kThreads),
                      smem_bytes(a.dim, a.vdim), stream, mq, mk, mv, p);
}

}  // namespace tllm
