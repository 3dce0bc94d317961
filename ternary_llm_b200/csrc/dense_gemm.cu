// Dense BF16 GEMM on the 5th-generation tensor cores (sm_100a): Y[M, N] = X[M, K] . W[N, K]^T
// with FP32 accumulation in tensor memory and the element-wise tail of the operator (bias,
// activation, gated product, per-head gate) in the epilogue.
//
// One CTA computes 128 tokens x TN features.  Both operands are K-major tiles of 64 columns
// brought by TMA with the 128-byte swizzle (out-of-range rows and columns read as zero, so no
// size needs to divide a tile); one thread issues tcgen05.mma kind::f16 (M = 128, N = TN,
// K = 16); a TMEM lane is a token, so an epilogue thread owns a token and writes runs of
// adjacent features.  A gated feed-forward loads TN/2 gate rows and the TN/2 up rows with the
// same numbers into one tile, so both factors of a product meet in the same thread.
// blockIdx.z walks the entries of a block-diagonal or per-head product (column offset in X and
// Y, row offset in W).  All mbarrier waits are bounded; a wait that gives up sets the device
// error flag, the roles wait for their own copies and MMAs (bounded again), and TMEM is freed.
#include <mutex>

#include "dense.cuh"
#include "launch.cuh"
#include "tcgen05.cuh"

namespace tllm {

namespace {

using namespace gemm;

constexpr int kTok = 128;            // tokens per CTA (MMA M, TMEM lanes)
constexpr int kBlkK = 64;            // K per stage: one 128-byte swizzled row
constexpr int kThr = 256;

template <int TN>
struct DCfg {
    static constexpr int kXBytes = kTok * kBlkK * 2;
    static constexpr int kWBytes = TN * kBlkK * 2;
    static constexpr int kStage = kXBytes + kWBytes;
    static constexpr int kStages = (TN == 256) ? 4 : (TN == 128) ? 3 : 4;
    static constexpr int kPerSm = (TN == 256) ? 1 : 2;
    static constexpr size_t kSmem = (size_t)kStages * kStage + 1024;
};

struct DenseEpi {
    void* y;
    const float* bias;
    const bf16* gate;
    int ldy, y_batch, gate_ld;
    int M, N, K, x_batch, w_rows;
    int act, glu, y_f32, vec;
    int* err;
};

template <int TN>
__device__ __forceinline__ uint32_t idesc_bf16()
{
    return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(TN >> 3) << 17) | ((uint32_t)(kTok >> 4) << 24);
}

__device__ __forceinline__ void mma_ss(uint32_t d, uint64_t a, uint64_t b, uint32_t idesc, uint32_t acc)
{
    asm volatile(
        "{ .reg .pred p; setp.ne.b32 p, %4, 0;\n"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p; }"
        ::"r"(d), "l"(a), "l"(b), "r"(idesc), "r"(acc) : "memory");
}

template <int TN>
__global__ void __launch_bounds__(kThr, DCfg<TN>::kPerSm)
dense_gemm_kernel(const __grid_constant__ CUtensorMap map_x, const __grid_constant__ CUtensorMap map_w, const DenseEpi a)
{
    constexpr int kStages = DCfg<TN>::kStages, kStage = DCfg<TN>::kStage, kXBytes = DCfg<TN>::kXBytes;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    __shared__ __align__(8) uint64_t bars[2 * kStages + 1];
    __shared__ uint32_t tmem_slot;
    __shared__ int abort_flag;
    pdl_launch_dependents();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int m0 = blockIdx.x * kTok, z = blockIdx.z;
    const int outs = a.glu ? TN / 2 : TN;              // output features of this tile
    const int n0 = blockIdx.y * outs;
    const int nk = (a.K + kBlkK - 1) / kBlkK;
    const uint32_t bar0 = smem_u32(bars);
    auto full = [&](int s) { return bar0 + 8u * s; };
    auto empty = [&](int s) { return bar0 + 8u * (kStages + s); };
    const uint32_t done = bar0 + 8u * (2 * kStages);

    if (tid == 0) {
        for (int s = 0; s < kStages; s++) {
            mbar_init(full(s), 1);
            mbar_init(empty(s), 1);
        }
        mbar_init(done, 1);
        abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;"
                     ::"r"(smem_u32(&tmem_slot)), "r"(TN) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = tmem_slot;
    volatile int* abortp = &abort_flag;
    pdl_wait();

    if (warp == 0) {
        if (lane == 0) {
            const int wr0 = z * a.w_rows + n0, wr1 = a.glu ? wr0 + a.N : wr0 + TN / 2;
            int it = 0;
            for (; it < nk; it++) {
                const int s = it % kStages;
                if (!mbar_wait(empty(s), ((it / kStages) & 1) ^ 1, abortp)) { abort_flag = 1; break; }
                mbar_expect_tx(full(s), kStage);
                const uint32_t dst = smem_u32(smem + (size_t)s * kStage);
                tma_load_2d(dst, &map_x, z * a.x_batch + it * kBlkK, m0, full(s));
                tma_load_2d(dst + kXBytes, &map_w, it * kBlkK, wr0, full(s));
                tma_load_2d(dst + kXBytes + TN / 2 * kBlkK * 2, &map_w, it * kBlkK, wr1, full(s));
            }
            // normally the MMAs have consumed every stage; after an abort the copies still in
            // flight must land before the shared memory goes away
            if (it < nk || *abortp) {
                int never = 0;
                for (int j = it > kStages ? it - kStages : 0; j < it; j++) mbar_wait(full(j % kStages), (j / kStages) & 1, &never);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t idesc = idesc_bf16<TN>();
            for (int it = 0; it < nk; it++) {
                const int s = it % kStages;
                if (!mbar_wait(full(s), (it / kStages) & 1, abortp)) { abort_flag = 1; break; }
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const uint32_t xb = smem_u32(smem + (size_t)s * kStage), wb = xb + kXBytes;
#pragma unroll
                for (int k = 0; k < kBlkK / 16; k++)
                    mma_ss(tmem, make_sw128_desc(xb + k * 32), make_sw128_desc(wb + k * 32), idesc, (it > 0 || k > 0) ? 1u : 0u);
                mma_commit(empty(s));
            }
            mma_commit(done);
            int never = 0;
            if (!mbar_wait(done, 0, &never)) abort_flag = 1;
        }
    } else if (warp >= 4) {
        const int row = tid - 128, m = m0 + row;
        int never = 0;
        // `done` arrives on every path of the issuer, an aborted one included
        const bool ok = __all_sync(0xffffffffu, mbar_wait(done, 0, &never) && !*abortp);
        if (ok) {
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const uint32_t lane_base = tmem + ((uint32_t)(row & ~31) << 16);
            const float hg = (a.gate && m < a.M) ? sigmoid_f(__bfloat162float(a.gate[(size_t)m * a.gate_ld + z])) : 1.f;
#pragma unroll 1
            for (int c = 0; c < outs; c += 32) {
                if (n0 + c >= a.N) break;
                uint32_t v[32];
                __syncwarp();
                tmem_ld32(lane_base + c, v);
                float f[32];
                if (a.glu) {
                    uint32_t u[32];
                    tmem_ld32(lane_base + TN / 2 + c, u);
                    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
                    for (int j = 0; j < 32; j++) f[j] = apply_act(a.act, __uint_as_float(v[j])) * __uint_as_float(u[j]);
                } else {
                    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
                    for (int j = 0; j < 32; j++) f[j] = __uint_as_float(v[j]);
                    if (a.bias) {
                        const float* b = a.bias + (size_t)z * a.N + n0 + c;
#pragma unroll
                        for (int j = 0; j < 32; j++)
                            if (n0 + c + j < a.N) f[j] += __ldg(b + j);
                    }
                    if (a.act != kActNone) {
#pragma unroll
                        for (int j = 0; j < 32; j++) f[j] = apply_act(a.act, f[j]);
                    }
                    if (a.gate) {
#pragma unroll
                        for (int j = 0; j < 32; j++) f[j] *= hg;
                    }
                }
                if (m >= a.M) continue;
                const size_t o = (size_t)m * a.ldy + (size_t)z * a.y_batch + n0 + c;
                if (a.vec && n0 + c + 32 <= a.N) {
                    if (a.y_f32) {
                        float4* p = reinterpret_cast<float4*>(static_cast<float*>(a.y) + o);
#pragma unroll
                        for (int j = 0; j < 8; j++) p[j] = make_float4(f[4 * j], f[4 * j + 1], f[4 * j + 2], f[4 * j + 3]);
                    } else {
                        uint4* p = reinterpret_cast<uint4*>(static_cast<bf16*>(a.y) + o);
#pragma unroll
                        for (int j = 0; j < 4; j++) {
                            uint32_t w[4];
#pragma unroll
                            for (int q = 0; q < 4; q++) {
                                const __nv_bfloat162 t = __floats2bfloat162_rn(f[8 * j + 2 * q], f[8 * j + 2 * q + 1]);
                                w[q] = *reinterpret_cast<const uint32_t*>(&t);
                            }
                            p[j] = make_uint4(w[0], w[1], w[2], w[3]);
                        }
                    }
                } else {
#pragma unroll
                    for (int j = 0; j < 32; j++) {
                        if (n0 + c + j >= a.N) continue;
                        if (a.y_f32) static_cast<float*>(a.y)[o + j] = f[j];
                        else static_cast<bf16*>(a.y)[o + j] = __float2bfloat16_rn(f[j]);
                    }
                }
            }
        } else {
            abort_flag = 1;
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (abort_flag && tid == 0) atomicExch(a.err, TLLM_ERR_TIMEOUT);
    if (warp == 1) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(TN) : "memory");
    }
}

int encode(EncodeTiledFn enc, CUtensorMap* map, const bf16* p, int cols, int rows, int ld, int box_rows)
{
    const cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
    const cuuint64_t strides[1] = {(cuuint64_t)ld * sizeof(bf16)};
    const cuuint32_t box[2] = {(cuuint32_t)kBlkK, (cuuint32_t)box_rows};
    const cuuint32_t estr[2] = {1, 1};
    const CUresult r = enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<bf16*>(p), dims, strides, box, estr,
                           CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
                           CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) return fail(TLLM_ERR_LAUNCH, "dense_gemm: cuTensorMapEncodeTiled failed with %d", (int)r);
    return TLLM_OK;
}

template <int TN>
int launch_tn(EncodeTiledFn enc, const LinearArgs<bf16>& l, DenseEpi e, cudaStream_t stream)
{
    CUtensorMap mx, mw;
    int st;
    if ((st = encode(enc, &mx, l.x, (l.batch - 1) * l.x_batch + l.K, l.M, l.ldx, kTok))) return st;
    if ((st = encode(enc, &mw, l.w, l.K, l.batch * l.w_rows, l.ldw, TN / 2))) return st;
    static bool attr[64] = {};
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev >= 0 && dev < 64 && !attr[dev]) {
        cudaFuncSetAttribute(dense_gemm_kernel<TN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)DCfg<TN>::kSmem);
        attr[dev] = true;
    }
    const int outs = l.glu ? TN / 2 : TN;
    return launch_pdl("dense_gemm", dense_gemm_kernel<TN>, dim3((l.M + kTok - 1) / kTok, (l.N + outs - 1) / outs, l.batch),
                      dim3(kThr), DCfg<TN>::kSmem, stream, mx, mw, e);
}

}  // namespace

int launch_dense_gemm_tcgen05(const LinearArgs<bf16>& l, cudaStream_t stream)
{
    if (l.M == 0 || l.N == 0 || l.batch == 0) return TLLM_OK;
    // K offsets of a TMA box must start on 16-byte boundaries, rows as well
    if (l.K < 8 || l.K % 8 || l.ldw % 8 || l.ldx % 8 || l.x_batch % 8)
        return fail(TLLM_ERR_SHAPE, "dense_gemm: K=%d ldw=%d ldx=%d x_batch=%d must be multiples of 8", l.K, l.ldw, l.ldx, l.x_batch);
    if ((reinterpret_cast<uintptr_t>(l.x) | reinterpret_cast<uintptr_t>(l.w)) & 15)
        return fail(TLLM_ERR_ALIGN, "dense_gemm: operands must be 16-byte aligned");
    if (l.w_rows < (l.glu ? 2 : 1) * l.N) return fail(TLLM_ERR_SHAPE, "dense_gemm: %d rows of W for N=%d", l.w_rows, l.N);
    EncodeTiledFn enc = encode_fn();
    if (!enc) return fail(TLLM_ERR_LAUNCH, "cuTensorMapEncodeTiled is not available from this driver");
    DenseEpi e = {};
    e.y = l.y;
    e.bias = l.bias;
    e.gate = l.gate;
    e.ldy = l.ldy;
    e.y_batch = l.y_batch;
    e.gate_ld = l.gate_ld;
    e.M = l.M;
    e.N = l.N;
    e.K = l.K;
    e.x_batch = l.x_batch;
    e.w_rows = l.w_rows;
    e.act = l.act;
    e.glu = l.glu;
    e.y_f32 = l.y_f32;
    const size_t es = l.y_f32 ? 4 : 2;
    e.vec = ((l.ldy * es) % 16 == 0 && (l.y_batch * es) % 16 == 0 && (reinterpret_cast<uintptr_t>(l.y) & 15) == 0);
    e.err = device_error_flag();
    if (!e.err) return fail(TLLM_ERR_LAUNCH, "device scratch unavailable");
    static int sms[64] = {};
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev < 0 || dev >= 64) return fail(TLLM_ERR_LAUNCH, "dense_gemm: no current device");
    if (!sms[dev]) cudaDeviceGetAttribute(&sms[dev], cudaDevAttrMultiProcessorCount, dev);
    // the widest tile that still gives most SMs one
    const long long mt = (l.M + kTok - 1) / kTok;
    auto tiles = [&](int tn) {
        const int outs = l.glu ? tn / 2 : tn;
        return mt * ((l.N + outs - 1) / outs) * l.batch;
    };
    if (tiles(256) * 10 >= 7LL * sms[dev]) return launch_tn<256>(enc, l, e, stream);
    if (tiles(128) * 10 >= 7LL * sms[dev]) return launch_tn<128>(enc, l, e, stream);
    return launch_tn<64>(enc, l, e, stream);
}

}  // namespace tllm
