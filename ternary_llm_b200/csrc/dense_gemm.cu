// Dense BF16 GEMM on the 5th-generation tensor cores (sm_100a): Y[M, N] = X[M, K] . W[N, K]^T
// with FP32 accumulation in tensor memory and the element-wise tail of the operator (bias,
// activation, gated product, per-head gate) in the epilogue.
//
// A tile is 128 tokens x TN features.  One persistent CTA per SM walks tiles with three roles
// that run ahead of one another: a TMA producer (K-major tiles of 64 columns, 128-byte swizzle;
// out-of-range rows and columns read as zero, so no size needs to divide a tile), one thread
// that issues tcgen05.mma kind::f16 (M = 128, N = TN, K = 16) into one of two accumulators in
// tensor memory, and eight epilogue warps that empty the other one: a TMEM lane is a token, the
// rows pass through a small shared-memory tile per warp so that global stores are whole lines.
// A gated feed-forward loads TN/2 gate rows and the TN/2 up rows with the same numbers into one
// tile, so both factors of a product meet in the same thread.  Tiles also run over the entries
// of a block-diagonal or per-head product (column offset in X and Y, row offset in W).  All
// mbarrier waits are bounded; a wait that gives up sets the device error flag, the roles wait
// for their own copies and MMAs (bounded again), and TMEM is freed.
#include <mutex>

#include "dense.cuh"
#include "launch.cuh"
#include "tcgen05.cuh"

namespace tllm {

namespace {

using namespace gemm;

constexpr int kTok = 128;            // tokens per CTA (MMA M, TMEM lanes)
constexpr int kBlkK = 64;            // K per stage: one 128-byte swizzled row
constexpr int kEpiWarps = 8;         // two per quarter of the TMEM lanes, taking turns at 32 columns
constexpr int kThr = 128 + 32 * kEpiWarps;

constexpr int kStageLd = 20;         // words per row of an epilogue warp's tile: 16 of data (16 FP32 or 32 BF16 columns)

template <int TN>
struct DCfg {
    static constexpr int kXBytes = kTok * kBlkK * 2;
    static constexpr int kWBytes = TN * kBlkK * 2;
    static constexpr int kStage = kXBytes + kWBytes;
    static constexpr int kStages = (TN == 256) ? 4 : (TN == 128) ? 6 : 8;
    static constexpr int kEpiBytes = kEpiWarps * 32 * kStageLd * 4;
    static constexpr size_t kSmem = (size_t)kStages * kStage + kEpiBytes + 1024;
};

struct DenseEpi {
    void* y;
    const float* bias;
    const bf16* gate;
    int ldy, y_batch, gate_ld;
    int M, N, K, x_batch, w_rows;
    int mt, nt, tiles;             // tiles along the tokens, along the features, in all
    int act, glu, y_f32, vec, bias_vec;
    float act_param;
    int act_lo, act_hi, f32_from, ldy2, vec2;
    float* y2;
    const int *group, *groups;
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
__global__ void __launch_bounds__(kThr, 1)
dense_gemm_kernel(const __grid_constant__ CUtensorMap map_x, const __grid_constant__ CUtensorMap map_w, const DenseEpi a)
{
    constexpr int kStages = DCfg<TN>::kStages, kStage = DCfg<TN>::kStage, kXBytes = DCfg<TN>::kXBytes;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    __shared__ __align__(8) uint64_t bars[2 * kStages + 4];
    __shared__ uint32_t tmem_slot;
    __shared__ int abort_flag;
    pdl_launch_dependents();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int outs = a.glu ? TN / 2 : TN;              // output features of a tile
    const int nk = (a.K + kBlkK - 1) / kBlkK;
    const uint32_t bar0 = smem_u32(bars);
    auto full = [&](int s) { return bar0 + 8u * s; };
    auto empty = [&](int s) { return bar0 + 8u * (kStages + s); };
    auto acc_full = [&](int i) { return bar0 + 8u * (2 * kStages + i); };
    auto acc_empty = [&](int i) { return bar0 + 8u * (2 * kStages + 2 + i); };

    if (tid == 0) {
        for (int s = 0; s < kStages; s++) {
            mbar_init(full(s), 1);
            mbar_init(empty(s), 1);
        }
        for (int i = 0; i < 2; i++) {
            mbar_init(acc_full(i), 1);
            mbar_init(acc_empty(i), 32 * kEpiWarps);
        }
        abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;"
                     ::"r"(smem_u32(&tmem_slot)), "r"(2 * TN) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = tmem_slot;
    volatile int* abortp = &abort_flag;
    int never = 0;
    pdl_wait();
    // tile -> first token, first feature, batch entry, entry of W; tokens vary fastest (neighbours
    // share W), with grouped rows those of one entry
    const int tiles = a.group ? min(*a.groups, a.mt) * a.nt : a.tiles;
    auto where = [&](int tile, int& m0, int& n0, int& z, int& entry) {
        if (a.group) {
            const int* g = a.group + 3 * (tile / a.nt);
            const int first = g[1], count = g[2], r = tile - first * a.nt, n = r / count;
            m0 = (first + r - n * count) * kTok;
            n0 = n * outs;
            z = 0;
            entry = g[0];
            return;
        }
        m0 = (tile % a.mt) * kTok;
        tile /= a.mt;
        n0 = (tile % a.nt) * outs;
        entry = z = tile / a.nt;
    };

    if (warp == 0) {
        // ---------------- TMA producer ----------------
        if (lane == 0) {
            int it = 0;                                  // stages filled so far, over all tiles
            bool ok = true;
            for (int tile = blockIdx.x; ok && tile < tiles; tile += gridDim.x) {
                int m0, n0, z, entry;
                where(tile, m0, n0, z, entry);
                const int wr0 = entry * a.w_rows + n0, wr1 = a.glu ? wr0 + a.N : wr0 + TN / 2;
                for (int k = 0; k < nk; k++, it++) {
                    const int s = it % kStages;
                    if (!mbar_wait(empty(s), ((it / kStages) & 1) ^ 1, abortp)) {
                        abort_flag = 1;
                        ok = false;
                        break;
                    }
                    mbar_expect_tx(full(s), kStage);
                    const uint32_t dst = smem_u32(smem + (size_t)s * kStage);
                    tma_load_2d(dst, &map_x, z * a.x_batch + k * kBlkK, m0, full(s));
                    tma_load_2d(dst + kXBytes, &map_w, k * kBlkK, wr0, full(s));
                    tma_load_2d(dst + kXBytes + TN / 2 * kBlkK * 2, &map_w, k * kBlkK, wr1, full(s));
                }
            }
            // normally the MMAs consume every stage; after an abort the copies still in flight
            // must land before the shared memory goes away
            if (*abortp)
                for (int j = it > kStages ? it - kStages : 0; j < it; j++) mbar_wait(full(j % kStages), (j / kStages) & 1, &never);
        }
    } else if (warp == 1) {
        // ---------------- MMA issuer ----------------
        if (lane == 0) {
            const uint32_t idesc = idesc_bf16<TN>();
            int it = 0, i = 0;                           // i: tiles of this CTA so far
            bool ok = true;
            for (int tile = blockIdx.x; ok && tile < tiles; tile += gridDim.x, i++) {
                const int buf = i & 1;
                if (!mbar_wait(acc_empty(buf), ((i >> 1) & 1) ^ 1, abortp)) {
                    abort_flag = 1;
                    break;
                }
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const uint32_t acc = tmem + buf * TN;
                for (int k = 0; k < nk; k++, it++) {
                    const int s = it % kStages;
                    if (!mbar_wait(full(s), (it / kStages) & 1, abortp)) {
                        abort_flag = 1;
                        ok = false;
                        break;
                    }
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                    const uint32_t xb = smem_u32(smem + (size_t)s * kStage), wb = xb + kXBytes;
#pragma unroll
                    for (int kk = 0; kk < kBlkK / 16; kk++)
                        mma_ss(acc, make_sw128_desc(xb + kk * 32), make_sw128_desc(wb + kk * 32), idesc, (k > 0 || kk > 0) ? 1u : 0u);
                    mma_commit(empty(s));
                }
                // arrives after everything issued so far, on the abort path too
                mma_commit(acc_full(buf));
            }
            // the last accumulators complete before TMEM and shared memory are given up
            for (int j = i > 2 ? i - 2 : 0; j < i; j++)
                if (!mbar_wait(acc_full(j & 1), (j >> 1) & 1, &never)) abort_flag = 1;
        }
    } else if (warp >= 4) {
        // ---------------- epilogue ----------------
        const int ew = warp - 4, row0 = (ew & 3) * 32, half = ew >> 2;
        const uint32_t lane_base = tmem + ((uint32_t)row0 << 16);
        uint32_t* st = reinterpret_cast<uint32_t*>(smem + (size_t)kStages * kStage) + ew * 32 * kStageLd;
        const int sr = lane >> 2, sw = (lane & 3) * 4;   // row (of eight) and words this lane stores
        int i = 0;
        for (int tile = blockIdx.x; tile < tiles; tile += gridDim.x, i++) {
            const int buf = i & 1;
            if (!__all_sync(0xffffffffu, mbar_wait(acc_full(buf), (i >> 1) & 1, abortp))) {
                abort_flag = 1;
                break;
            }
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            int m0, n0, z, entry;
            where(tile, m0, n0, z, entry);
            const int mrow = m0 + row0;
            const float hg = (a.gate && mrow + lane < a.M) ? sigmoid_f(__bfloat162float(a.gate[(size_t)(mrow + lane) * a.gate_ld + z])) : 1.f;
            const int ncols = min(outs, a.N - n0);
            const uint32_t acc = lane_base + buf * TN;
            if (mrow < a.M)
#pragma unroll 1
            for (int c = half * 32; c < ncols; c += 64) {
                // 32 columns go one way: the limits of the activation and of y2 are multiples of 64
                const bool second = n0 + c >= a.f32_from, y_f32 = a.y_f32 || second;
                const int act = n0 + c >= a.act_lo && n0 + c < a.act_hi && !second ? a.act : kActNone;
                const int wcols = y_f32 ? 1 : 2;         // columns per staged word
                uint32_t v[32];
                __syncwarp();
                tmem_ld32(acc + c, v);
                float f[32];
                if (a.glu) {
                    uint32_t u[32];
                    tmem_ld32(acc + TN / 2 + c, u);
                    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
                    for (int j = 0; j < 32; j++) f[j] = __uint_as_float(v[j]);
                    apply_act_n<32>(act, f);
#pragma unroll
                    for (int j = 0; j < 32; j++) f[j] *= __uint_as_float(u[j]);
                } else {
                    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
                    for (int j = 0; j < 32; j++) f[j] = __uint_as_float(v[j]);
                    if (a.bias) {
                        const float* bp = a.bias + (size_t)z * a.N + n0 + c;
                        if (a.bias_vec && c + 32 <= ncols) {
#pragma unroll
                            for (int j = 0; j < 8; j++) {
                                const float4 t = __ldg(reinterpret_cast<const float4*>(bp) + j);
                                f[4 * j] += t.x;
                                f[4 * j + 1] += t.y;
                                f[4 * j + 2] += t.z;
                                f[4 * j + 3] += t.w;
                            }
                        } else {
#pragma unroll
                            for (int j = 0; j < 32; j++)
                                if (c + j < ncols) f[j] += __ldg(bp + j);
                        }
                    }
                    apply_act_n<32>(act, f, a.act_param);
                    if (a.gate) {
#pragma unroll
                        for (int j = 0; j < 32; j++) f[j] *= hg;
                    }
                }
                // through shared memory, 16 words of a row at a time: FP32 in two halves, BF16 at once
#pragma unroll
                for (int part = 0; part < 2; part++) {
                    if (part == 1 && !y_f32) break;
                    __syncwarp();
#pragma unroll
                    for (int j = 0; j < 4; j++) {
                        uint32_t w[4];
#pragma unroll
                        for (int q = 0; q < 4; q++) {
                            const int e = 4 * j + q;
                            if (y_f32) {
                                w[q] = __float_as_uint(f[part * 16 + e]);
                            } else {
                                const __nv_bfloat162 t = __floats2bfloat162_rn(f[2 * e], f[2 * e + 1]);
                                w[q] = *reinterpret_cast<const uint32_t*>(&t);
                            }
                        }
                        *reinterpret_cast<uint4*>(st + lane * kStageLd + 4 * j) = make_uint4(w[0], w[1], w[2], w[3]);
                    }
                    __syncwarp();
                    const int col = c + part * 16 + sw * wcols;      // first of this lane's columns inside the tile
                    if (col < ncols) {
                        const bool vec = (second ? a.vec2 : a.vec) && col + 4 * wcols <= ncols;
#pragma unroll
                        for (int r = 0; r < 4; r++) {
                            const int rr = r * 8 + sr, m = mrow + rr;
                            if (m >= a.M) break;
                            const uint4 t = *reinterpret_cast<const uint4*>(st + rr * kStageLd + sw);
                            const size_t o = second ? (size_t)m * a.ldy2 + n0 + col - a.f32_from
                                                    : (size_t)m * a.ldy + (size_t)z * a.y_batch + n0 + col;
                            if (vec) {
                                if (y_f32) *reinterpret_cast<uint4*>((second ? a.y2 : static_cast<float*>(a.y)) + o) = t;
                                else *reinterpret_cast<uint4*>(static_cast<bf16*>(a.y) + o) = t;
                            } else {
                                const uint32_t w[4] = {t.x, t.y, t.z, t.w};
                                for (int q = 0; q < 4 * wcols && col + q < ncols; q++) {
                                    if (y_f32) (second ? a.y2 : static_cast<float*>(a.y))[o + q] = __uint_as_float(w[q]);
                                    else static_cast<uint16_t*>(a.y)[o + q] = (uint16_t)(w[q >> 1] >> ((q & 1) * 16));
                                }
                            }
                        }
                    }
                }
            }
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            mbar_arrive(acc_empty(buf));
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (abort_flag && tid == 0) atomicExch(a.err, TLLM_ERR_TIMEOUT);
    if (warp == 1) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(2 * TN) : "memory");
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
int launch_tn(EncodeTiledFn enc, const LinearArgs<bf16>& l, DenseEpi e, int sms, cudaStream_t stream)
{
    CUtensorMap mx, mw;
    int st;
    if ((st = encode(enc, &mx, l.x, (l.batch - 1) * l.x_batch + l.K, l.M, l.ldx, kTok))) return st;
    if ((st = encode(enc, &mw, l.w, l.K, (l.group ? l.entries : l.batch) * l.w_rows, l.ldw, TN / 2))) return st;
    static bool attr[64] = {};
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev >= 0 && dev < 64 && !attr[dev]) {
        cudaFuncSetAttribute(dense_gemm_kernel<TN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)DCfg<TN>::kSmem);
        attr[dev] = true;
    }
    const int outs = l.glu ? TN / 2 : TN;
    e.mt = (l.M + kTok - 1) / kTok;
    e.nt = (l.N + outs - 1) / outs;
    e.tiles = e.mt * e.nt * l.batch;
    return launch_pdl("dense_gemm", dense_gemm_kernel<TN>, dim3(e.tiles < sms ? e.tiles : sms), dim3(kThr), DCfg<TN>::kSmem, stream, mx, mw, e);
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
    if (l.group && (l.batch != 1 || !l.groups)) return fail(TLLM_ERR_SHAPE, "dense_gemm: grouped rows with %d batch entries", l.batch);
    if ((l.act_lo | (l.act_hi == INT_MAX ? 0 : l.act_hi) | (l.f32_from == INT_MAX ? 0 : l.f32_from)) % 64 ||
        ((l.act_lo || l.act_hi != INT_MAX || l.f32_from != INT_MAX) && (l.glu || l.batch != 1)))
        return fail(TLLM_ERR_SHAPE, "dense_gemm: column ranges %d..%d and %d", l.act_lo, l.act_hi, l.f32_from);
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
    e.bias_vec = l.N % 4 == 0 && (reinterpret_cast<uintptr_t>(l.bias) & 15) == 0;
    e.act_param = l.act_param;
    e.act_lo = l.act_lo;
    e.act_hi = l.act_hi;
    e.f32_from = l.f32_from;
    e.y2 = l.y2;
    e.ldy2 = l.ldy2;
    e.vec2 = l.ldy2 % 4 == 0 && (reinterpret_cast<uintptr_t>(l.y2) & 15) == 0;
    e.group = l.group;
    e.groups = l.groups;
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
    if (tiles(256) * 10 >= 7LL * sms[dev]) return launch_tn<256>(enc, l, e, sms[dev], stream);
    if (tiles(128) * 10 >= 7LL * sms[dev]) return launch_tn<128>(enc, l, e, sms[dev], stream);
    return launch_tn<64>(enc, l, e, sms[dev], stream);
}

}  // namespace tllm
