// Recurrences whose state is a matrix per head: the gated delta rule and linear attention with a
// constant decay (equations in mixers.cuh), and the gated norm behind them.
//
// Token by token (decode, short portions, the exact 32-bit mode): a column of the state is held
// in the registers of a few lanes.
//
// Many tokens (BF16): chunks of 64 tokens, the products on tensor cores.  Inside a chunk with
// starting state S0, running decay G_i = g_1 .. g_i and unit vectors k_i, q_i,
//   (1 + A) U = beta (V - G K S0),  A_ij = beta_i (G_i / G_j) k_i.k_j  (j < i)
//   O = G Q S0 + P U,               P_ij = (G_i / G_j) q_i.k_j         (j <= i)
//   S = G_64 S0 + K^T (G_64 / G_j) U
// (the delta rule's updates of a chunk written as one triangular system; linear attention is
// U = V).  A first launch computes (1 + A)^-1 and P for all chunks at once, a second one walks the
// chunks with a slice of the state's columns per CTA.  Projected vectors enter the products
// as the BF16 numbers they are; their norms, decays and step sizes stay FP32 factors outside the
// products; the FP32 operands (state, U, P, the inverse) enter as the sum of two BF16 numbers.
#include "launch.cuh"
#include "matrix_step.cuh"
#include "mixers.cuh"
#include "mma_sync.cuh"
#include "tcgen05.cuh"

namespace tllm {

namespace {

// ---------------------------------------------------------------------------
// Chunks
// ---------------------------------------------------------------------------
constexpr int kC = 64, kChunkThreads = 256;
constexpr int kLdC = kC + 8;                       // row stride of a [64][64] tile in shared memory
constexpr int kLdA = kC + 4;                       // of an FP32 one

// floats of the region that holds the queries, then the inverse
__host__ __device__ inline int inverse_floats(int ld) { return kC * (ld / 2 > kLdA ? ld / 2 : kLdA); }

// What the first launch leaves for the second, laid out as it lies in shared memory there, so that a
// tile is one bulk copy.  Per (sequence, chunk, key head): keys, then queries, [64][ld], zero behind
// the sequence; per (sequence, chunk, head): slices of `nv` value columns [64][nv + 8]; matrices
// [64][kLdC], BF16 high and low parts -- P, then with the delta
// rule the inverse -- and four vectors of 64 floats (log of the running decay, step size, 1/|k|,
// q_scale/|q|)
struct ChunkWs {
    bf16 *kq, *v, *mats;
    float *vecs, *rec;
    int n_mats, nv;
    int* err;
};
__device__ __forceinline__ void bulk_copy(void* dst, const void* src, uint32_t bytes, uint32_t bar)
{
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                 ::"r"(sm32(dst)), "l"(src), "r"(bytes), "r"(bar) : "memory");
}
template <int THREADS>
__device__ __forceinline__ void carriers_sync() { asm volatile("bar.sync 1, %0;" ::"n"(THREADS) : "memory"); }
constexpr int kThreadsPerCol = 16;                 // scan: carriers and outputs, 4 warps per group of 16 columns each
__host__ __device__ inline size_t chunk_mats(bool delta) { return delta ? 4 : 2; }
inline int chunks_of(int n) { return (n + kC - 1) / kC; }

template <bool DELTA>
__global__ void __launch_bounds__(kChunkThreads)
chunk_prepare_kernel(const MatrixScanArgs<bf16> a, ChunkWs ws)
{
    extern __shared__ __align__(16) uint8_t smem_raw[];
    const int D = a.dim, ld = ((D + 15) & ~15) + 8, ksteps = (D + 15) / 16;
    // keys [64][ld], queries [64][ld]; delta: A [64][kLdA], a block column of sums, and the inverse
    // [64][kLdA] over the queries
    bf16* ks = reinterpret_cast<bf16*>(smem_raw);
    bf16* qs = ks + kC * ld;
    float* inv = reinterpret_cast<float*>(qs);
    float* A = inv + inverse_floats(ld);
    float* tmp = A + kC * kLdA;
    __shared__ float logg[kC], beta[kC], rk[kC], rq[kC];
    pdl_launch_dependents();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int chunk = blockIdx.x, h = blockIdx.y, b = blockIdx.z, kh = h / (a.heads / a.kv_heads);
    const int n = min(kC, a.g.seq_len - chunk * kC);
    const size_t row0 = (size_t)b * a.g.seq_len + (size_t)chunk * kC;
    const size_t unit = ((size_t)b * gridDim.x + chunk) * a.heads + h;
    bf16* mats = ws.mats + unit * ws.n_mats * kC * kLdC;
    pdl_wait();
    {
        const int pieces = D / 8, per = ld / 8;
        for (int r = warp; r < kC; r += kChunkThreads / 32)
            for (int c = lane; c < per; c += 32) {
                const bool v = r < n && c < pieces;
                const size_t o = (row0 + (v ? r : 0)) * a.ld + (size_t)kh * D + (v ? c * 8 : 0);
                cp16(ks + r * ld + c * 8, a.k + o, v);
                cp16(qs + r * ld + c * 8, a.q + o, v);
            }
        cp_commit();
    }
    if (DELTA && warp == 0) {
        float lg[2];
#pragma unroll
        for (int u = 0; u < 2; u++) {
            const int t = 2 * lane + u;
            lg[u] = t < n ? log_decay(a.a[(row0 + t) * a.ld_ab + h], a.dt_bias[h], a.neg_a[h]) : 0.f;
            beta[t] = t < n ? sigmoid_f(a.b[(row0 + t) * a.ld_ab + h]) : 0.f;
        }
        float s = lg[0] + lg[1];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float v = __shfl_up_sync(0xffffffffu, s, o);
            if (lane >= o) s += v;
        }
        logg[2 * lane] = s - lg[1];
        logg[2 * lane + 1] = s;
    }
    {
        const int slices = (a.vdim + ws.nv - 1) / ws.nv, per = ws.nv / 8, ldv = ws.nv + 8;
        bf16* v = ws.v + unit * slices * kC * ldv;
        const int shift = per == 2 ? 1 : 2;
        for (int r = warp; r < kC; r += kChunkThreads / 32)
            for (int c = lane; c < slices * per; c += 32) {
                const uint4 x = (r < n && c * 8 < a.vdim) ? *(reinterpret_cast<const uint4*>(a.v + (row0 + r) * a.ld + (size_t)h * a.vdim) + c)
                                                          : make_uint4(0, 0, 0, 0);
                const int s = c >> shift;
                *reinterpret_cast<uint4*>(v + (s * kC + r) * ldv + (c - s * per) * 8) = x;
            }
    }
    cp_wait<0>();
    __syncthreads();
    if (h % (a.heads / a.kv_heads) == 0) {
        uint4* kq = reinterpret_cast<uint4*>(ws.kq + (((size_t)b * gridDim.x + chunk) * a.kv_heads + kh) * 2 * kC * ld);
        for (int i = tid; i < 2 * kC * ld / 8; i += kChunkThreads) kq[i] = reinterpret_cast<const uint4*>(ks)[i];
    }
    if (DELTA) {
        // a quarter of a warp per vector
        for (int i = tid >> 3; i < 2 * kC; i += kChunkThreads / 8) {
            const bf16* x = (i < kC ? ks : qs) + (i & (kC - 1)) * ld;
            float ss = 0.f;
            for (int c = (tid & 7) * 8; c < D; c += 64) {
                float f[8];
                Vec16<bf16>::unpack(*reinterpret_cast<const uint4*>(x + c), f);
#pragma unroll
                for (int j = 0; j < 8; j++) ss += f[j] * f[j];
            }
            ss += __shfl_xor_sync(0xffffffffu, ss, 1);
            ss += __shfl_xor_sync(0xffffffffu, ss, 2);
            ss += __shfl_xor_sync(0xffffffffu, ss, 4);
            if ((tid & 7) == 0) {
                const float f = 1.f / sqrtf(ss + kUnitEps);
                if (i < kC) rk[i] = f;
                else rq[i - kC] = f * a.q_scale;
            }
        }
    } else if (tid < kC) {
        const float d = a.decay[h];
        logg[tid] = (float)(tid + 1) * (d > 0.f ? logf(d) : -100.f);
        rk[tid] = rq[tid] = 1.f;
    }
    __syncthreads();
    if (tid < kC) {
        float* v = ws.vecs + unit * 4 * kC + tid;
        v[0] = logg[tid];
        v[kC] = DELTA ? beta[tid] : 0.f;
        v[2 * kC] = rk[tid];
        v[3 * kC] = rq[tid];
    }
    // 16 rows of X K^T: sums of columns 0 .. 16 * (rows / 16 + 1)
    auto gram = [&](const bf16* x, int r0, float (&s)[8][4]) {
#pragma unroll
        for (int j = 0; j < 8; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) s[j][e] = 0.f;
        for (int k = 0; k < ksteps; k++) {
            uint32_t fa[4];
            ldsm4(fa, x + (r0 + (lane & 15)) * ld + k * 16 + (lane >> 4) * 8);
#pragma unroll
            for (int j = 0; j < 8; j += 2) {
                if (j * 8 > r0) break;
                uint32_t fb[4];
                ldsm4(fb, ks + (j * 8 + (lane & 7) + (lane >> 4) * 8) * ld + k * 16 + ((lane >> 3) & 1) * 8);
                mma16816(s[j], fa, fb[0], fb[1]);
                mma16816(s[j + 1], fa, fb[2], fb[3]);
            }
        }
    };
    auto weight = [&](int i, int j) { return exp2_neg(1.4426950408889634f * (logg[i] - logg[j])); };   // G_i / G_j, j <= i
    auto write_p = [&](int r0) {
        float s[8][4];
        gram(qs, r0, s);
#pragma unroll
        for (int j = 0; j < 8; j++)
#pragma unroll
            for (int half = 0; half < 2; half++) {
                const int i = r0 + (lane >> 2) + half * 8, c = j * 8 + 2 * (lane & 3);
                float p[2];
#pragma unroll
                for (int e = 0; e < 2; e++) p[e] = c + e <= i ? s[j][2 * half + e] * weight(i, c + e) * rq[i] * rk[c + e] : 0.f;
                uint32_t hi, lo;
                split2(p[0], p[1], hi, lo);
                *reinterpret_cast<uint32_t*>(mats + i * kLdC + c) = hi;
                *reinterpret_cast<uint32_t*>(mats + kC * kLdC + i * kLdC + c) = lo;
            }
    };
    if (warp >= 4) write_p((warp - 4) * 16);
    if (!DELTA) return;
    if (warp < 4) {
        float s[8][4];
        gram(ks, warp * 16, s);
#pragma unroll
        for (int j = 0; j < 8; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int i = warp * 16 + (lane >> 2) + (e >> 1) * 8, c = j * 8 + 2 * (lane & 3) + (e & 1);
                A[i * kLdA + c] = c < i ? beta[i] * weight(i, c) * rk[i] * rk[c] * s[j][e] : 0.f;
            }
    }
    __syncthreads();                                        // A is there, and nobody reads the queries any more
    // (1 + A)^-1 by blocks of 16: the diagonal ones by substitution, a column per thread
    constexpr int kB = 16, nb = kC / kB;
    if (tid < kC) {
        const int d0 = tid & ~(kB - 1), col = tid & (kB - 1);
        float x[kB];
#pragma unroll
        for (int i = 0; i < kB; i++) {
            float v = i == col ? 1.f : 0.f;
#pragma unroll
            for (int j = 0; j < i; j++) v = fmaf(-A[(d0 + i) * kLdA + d0 + j], x[j], v);
            x[i] = v;
            inv[(d0 + i) * kLdA + d0 + col] = v;
        }
    } else {                                                // blocks above the diagonal are zero
        for (int i = tid - kC; i < kC * kC; i += kChunkThreads - kC) {
            const int r = i / kC, c = i % kC;
            if (r / kB < c / kB) inv[r * kLdA + c] = 0.f;
        }
    }
    __syncthreads();
    // then block (j + d, j) = -inv_ii sum_k A_ik inv_kj, one distance after the other: 64 threads per
    // block, 2 x 2 entries each
    const int j = tid >> 6, tr = (tid >> 3 & 7) * 2, tc = (tid & 7) * 2;
    auto tile_product = [&](const float* x, int ldx, const float* y, int ldy, int n, float2 (&v)[2]) {
        v[0] = v[1] = make_float2(0.f, 0.f);
#pragma unroll 8
        for (int k = 0; k < n; k++) {
            const float2 q = *reinterpret_cast<const float2*>(y + k * ldy + tc);
            const float p0 = x[tr * ldx + k], p1 = x[(tr + 1) * ldx + k];
            v[0].x = fmaf(p0, q.x, v[0].x);
            v[0].y = fmaf(p0, q.y, v[0].y);
            v[1].x = fmaf(p1, q.x, v[1].x);
            v[1].y = fmaf(p1, q.y, v[1].y);
        }
    };
    for (int d = 1; d < nb; d++) {
        float2 v[2];
        const int i0 = (j + d) * kB;
        if (j + d < nb) {
            tile_product(A + i0 * kLdA + j * kB, kLdA, inv + j * kB * kLdA + j * kB, kLdA, d * kB, v);
            *reinterpret_cast<float2*>(tmp + j * kB * kB + tr * kB + tc) = v[0];
            *reinterpret_cast<float2*>(tmp + j * kB * kB + (tr + 1) * kB + tc) = v[1];
        }
        __syncthreads();
        if (j + d < nb) {
            tile_product(inv + i0 * kLdA + i0, kLdA, tmp + j * kB * kB, kB, kB, v);
            *reinterpret_cast<float2*>(inv + (i0 + tr) * kLdA + j * kB + tc) = make_float2(-v[0].x, -v[0].y);
            *reinterpret_cast<float2*>(inv + (i0 + tr + 1) * kLdA + j * kB + tc) = make_float2(-v[1].x, -v[1].y);
        }
        __syncthreads();
    }
    for (int i = tid; i < kC * kC / 4; i += kChunkThreads) {
        const float4 v = *reinterpret_cast<const float4*>(inv + (i >> 4) * kLdA + (i & 15) * 4);
        uint32_t h0, l0, h1, l1;
        split2(v.x, v.y, h0, l0);
        split2(v.z, v.w, h1, l1);
        bf16* m = mats + 2 * kC * kLdC + (i >> 4) * kLdC + (i & 15) * 4;
        *reinterpret_cast<uint2*>(m) = make_uint2(h0, h1);
        *reinterpret_cast<uint2*>(m + kC * kLdC) = make_uint2(l0, l1);
    }
}

// A segment of the chunks and NV columns of the state per CTA.  Half of the warps carry the state
// (U, then the state behind the chunk), the others compute the outputs beside them; in each half
// four row tiles (of tokens; of the state MT each) times groups of 16 columns.  `stages` chunks are
// in flight.
//
// Linear attention is cut into segments that run at the same time: RECORD runs all but the last
// from a zero state and keeps their final states, the second launch starts each segment from the
// carried state and the records before it.  (The record of the last segment holds a copy of the
// carried state, which that segment overwrites while others may not have started.)
template <bool DELTA, int NV, int MT, bool RECORD>
__global__ void __launch_bounds__(kThreadsPerCol * NV)
chunk_scan_kernel(const MatrixScanArgs<bf16> a, ChunkWs ws, int nchunk, int per_seg, int nseg, int stages)
{
    extern __shared__ __align__(16) uint8_t smem_raw[];
    constexpr int kGroups = NV / 16, kThreads = kThreadsPerCol * NV, ldv = NV + 8, NT = 2, MATS = DELTA ? 4 : 2;
    const int D = a.dim, D16 = (D + 15) & ~15, ld = D16 + 8, ksteps = D16 / 16;
    const int tile = 2 * kC * ld + MATS * kC * kLdC + kC * ldv;               // bf16 of a stage, then 4 * 64 floats
    const size_t stage_bytes = (size_t)tile * 2 + 4 * kC * sizeof(float);
    bf16* sh = reinterpret_cast<bf16*>(smem_raw + stages * stage_bytes);       // state [D16][ldv], high and low
    bf16* rs = sh + 2 * D16 * ldv;                                             // right-hand side [64][ldv], high and low
    bf16* us = rs + (DELTA ? 2 * kC * ldv : 0);                                // U
    bf16* ups = us + (DELTA ? 2 * kC * ldv : 0);                               // U times its decay to the end
    __shared__ __align__(8) uint64_t full[2];
    __shared__ int abort_flag;
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, gq = lane >> 2, tq = lane & 3;
    const bool carrier = tid < kThreads / 2;                                   // carries the state
    // the triangular products grow with the row: the other way round in the two halves, which share schedulers
    const int warp = carrier ? tid >> 5 & 3 : 3 - (tid >> 5 & 3);
    const int n0 = (tid >> 7) % kGroups * NT * 8;                              // first column of the warp
    const int slices = (a.vdim + NV - 1) / NV, seg = blockIdx.x / slices;
    const int v0 = (blockIdx.x - seg * slices) * NV, h = blockIdx.y, b = blockIdx.z, kh = h / (a.heads / a.kv_heads);
    const int nv = min(NV, a.vdim - v0), c0 = seg * per_seg, c1 = min(nchunk, c0 + per_seg);
    const size_t row0 = (size_t)b * a.g.seq_len;
    int never = 0;
    if (tid == 0) {
        gemm::mbar_init(gemm::smem_u32(&full[0]), 1);
        gemm::mbar_init(gemm::smem_u32(&full[1]), 1);
        abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    pdl_wait();
    const bool fresh = (a.g.pos_dev ? *a.g.pos_dev : a.g.start_pos) == 0;
    float* st = a.state + (size_t)(a.g.first_slot + b) * a.slot_stride + ((size_t)h * a.vdim + v0) * D;
    const size_t rec_size = (size_t)a.heads * a.vdim * D;                      // of one segment
    float* rec = ws.rec + (size_t)b * nseg * rec_size + ((size_t)h * a.vdim + v0) * D;

    // the tiles of a chunk, by bulk copies that report to the stage's barrier
    auto request = [&](int c, int stage) {
        bf16* p = reinterpret_cast<bf16*>(smem_raw + stage * stage_bytes);
        const uint32_t bar = gemm::smem_u32(&full[stage]);
        const size_t unit = ((size_t)b * nchunk + c) * a.heads + h, kunit = ((size_t)b * nchunk + c) * a.kv_heads + kh;
        const uint32_t kq = (RECORD ? 1 : 2) * kC * ld * 2, m = RECORD ? 0 : MATS * kC * kLdC * 2, v = kC * ldv * 2, vec = 4 * kC * 4;
        gemm::mbar_expect_tx(bar, kq + m + v + vec);
        bulk_copy(p, ws.kq + kunit * 2 * kC * ld, kq, bar);
        if (!RECORD) bulk_copy(p + 2 * kC * ld, ws.mats + unit * MATS * kC * kLdC, m, bar);
        bulk_copy(p + 2 * kC * ld + MATS * kC * kLdC, ws.v + (unit * slices + v0 / NV) * kC * ldv, v, bar);
        bulk_copy(p + tile, ws.vecs + unit * 4 * kC, vec, bar);
    };
    const bool requester = tid == kThreads / 2;
    if (requester) request(c0, 0);

    float S[MT][NT][4];
    auto each_state = [&](auto&& f) {                       // (tile, column tile, element, row, column)
#pragma unroll
        for (int i = 0; i < MT; i++)
#pragma unroll
            for (int j = 0; j < NT; j++)
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const int r = (warp + 4 * i) * 16 + gq + (e >> 1) * 8, c = n0 + j * 8 + 2 * tq + (e & 1);
                    const bool in = r < D && c < nv;
                    f(S[i][j][e], in, in ? (size_t)c * D + r : 0);   // a place that may be read either way
                }
    };
    auto save_state = [&]() {                               // as two BF16 matrices
#pragma unroll
        for (int i = 0; i < MT; i++) {
            const int r = (warp + 4 * i) * 16 + gq;
            if ((warp + 4 * i) * 16 >= D16) break;
#pragma unroll
            for (int j = 0; j < NT; j++)
#pragma unroll
                for (int half = 0; half < 2; half++) {
                    uint32_t hi, lo;
                    split2(S[i][j][2 * half], S[i][j][2 * half + 1], hi, lo);
                    const int o = (r + half * 8) * ldv + n0 + j * 8 + 2 * tq;
                    *reinterpret_cast<uint32_t*>(sh + o) = hi;
                    *reinterpret_cast<uint32_t*>(sh + D16 * ldv + o) = lo;
                }
        }
    };
    if (carrier) {
        // loads without branches: all of them are in flight together
        const float keep = fresh ? 0.f : 1.f;
        if (RECORD || nseg == 1) each_state([&](float& x, bool in, size_t o) { const float v = st[o]; x = in && keep != 0.f ? v : 0.f; });
        if (RECORD) {
            if (seg == 0) each_state([&](float& x, bool in, size_t o) { if (in) rec[(size_t)(nseg - 1) * rec_size + o] = x; });
            each_state([&](float& x, bool, size_t) { x = 0.f; });
        } else if (nseg > 1) {
            each_state([&](float& x, bool in, size_t o) { const float v = rec[(size_t)(nseg - 1) * rec_size + o]; x = in ? v : 0.f; });
            const float d = DELTA ? 0.f : a.decay[h], f = expf((float)(per_seg * kC) * (d > 0.f ? logf(d) : -100.f));
#pragma unroll 2
            for (int k = 0; k < seg; k++)
                each_state([&](float& x, bool in, size_t o) { const float v = rec[(size_t)k * rec_size + o]; x = in ? fmaf(f, x, v) : 0.f; });
        }
        if (!RECORD) save_state();
    }
    const int lda = lane & 15, ldb = (lane >> 4) * 8;
    const int i0 = warp * 16 + gq;                          // this lane's rows i0 and i0 + 8 of a chunk
    auto zero = [](float (&x)[NT][4]) {
#pragma unroll
        for (int j = 0; j < NT; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) x[j][e] = 0.f;
    };
    auto join = [](float (&x)[NT][4], const float (&y)[NT][4]) {
#pragma unroll
        for (int j = 0; j < NT; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) x[j][e] += y[j][e];
    };
    // x += (16 rows of the matrix m, its columns 16 k ..) times rows 16 k .. of u
    auto times = [&](float (&x)[NT][4], const uint32_t (&f)[4], const bf16* u, int k) {
        uint32_t fb[4];
        ldsm4t(fb, u + (k * 16 + lda) * ldv + n0 + ldb);
        mma16816(x[0], f, fb[0], fb[1]);
        mma16816(x[1], f, fb[2], fb[3]);
    };

    bool ok = true;
    for (int c = c0; c < c1; c++) {
        const int stage = stages == 2 ? (c - c0) & 1 : 0, n = min(kC, a.g.seq_len - c * kC);
        const bf16* kt = reinterpret_cast<const bf16*>(smem_raw + stage * stage_bytes);
        const bf16 *qt = kt + kC * ld, *pm = qt + kC * ld, *tm = pm + 2 * kC * kLdC, *vt = pm + MATS * kC * kLdC;
        const float* logg = reinterpret_cast<const float*>(vt + kC * ldv);
        const float *beta = logg + kC, *rk = beta + kC, *rq = rk + kC;
        __syncthreads();                                    // the state is there, nobody reads the other stage any more
        if (requester && stages == 2 && c + 1 < c1) request(c + 1, stage ^ 1);
        const int turn = stages == 2 ? (c - c0) >> 1 : c - c0;
        if (ok && !gemm::mbar_wait(gemm::smem_u32(&full[stage]), turn & 1, &abort_flag)) {
            ok = false;                                     // the sums are wrong from here on, the loop ends all the same
            abort_flag = 1;
        }
        const float end = logg[n - 1];
        float acc[NT][4], low[NT][4], dec[2];               // two chains of sums: high parts, the rest
        zero(acc);
        zero(low);
#pragma unroll
        for (int half = 0; half < 2; half++) dec[half] = exp2_neg(1.4426950408889634f * logg[i0 + half * 8]);
        if (carrier) {
            float to_end[2];
#pragma unroll
            for (int half = 0; half < 2; half++) {
                const int i = i0 + half * 8;
                to_end[half] = i < n ? exp2_neg(1.4426950408889634f * (end - logg[i])) * rk[i] : 0.f;
            }
            if (DELTA) {
#pragma unroll 4
                for (int k = 0; k < ksteps; k++) {          // K S0
                    uint32_t f[4];
                    ldsm4(f, kt + (warp * 16 + lda) * ld + k * 16 + ldb);
                    times(acc, f, sh, k);
                    times(low, f, sh + D16 * ldv, k);
                }
                join(acc, low);
#pragma unroll
                for (int j = 0; j < NT; j++)
#pragma unroll
                    for (int half = 0; half < 2; half++) {
                        const int i = i0 + half * 8, o = i * ldv + n0 + j * 8 + 2 * tq;
                        const float f = dec[half] * rk[i], be = beta[i];
                        const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(vt + o));
                        uint32_t hi, lo;
                        split2(be * (v.x - f * acc[j][2 * half]), be * (v.y - f * acc[j][2 * half + 1]), hi, lo);
                        *reinterpret_cast<uint32_t*>(rs + o) = hi;
                        *reinterpret_cast<uint32_t*>(rs + kC * ldv + o) = lo;
                    }
                carriers_sync<kThreads / 2>();
                float mid[NT][4];
                zero(acc);
                zero(low);
                zero(mid);
                for (int k = 0; k <= warp; k++) {           // U, the inverse is triangular
                    uint32_t fh[4], fl[4];
                    ldsm4(fh, tm + (warp * 16 + lda) * kLdC + k * 16 + ldb);
                    ldsm4(fl, tm + kC * kLdC + (warp * 16 + lda) * kLdC + k * 16 + ldb);
                    times(acc, fh, rs, k);
                    times(low, fl, rs, k);
                    times(mid, fh, rs + kC * ldv, k);
                }
                join(low, mid);
                join(acc, low);
            }
#pragma unroll
            for (int j = 0; j < NT; j++)
#pragma unroll
                for (int half = 0; half < 2; half++) {
                    const int o = (i0 + half * 8) * ldv + n0 + j * 8 + 2 * tq;
                    float2 u;
                    uint32_t hi, lo;
                    if (DELTA) {
                        u = make_float2(acc[j][2 * half], acc[j][2 * half + 1]);
                        split2(u.x, u.y, hi, lo);
                        *reinterpret_cast<uint32_t*>(us + o) = hi;
                        *reinterpret_cast<uint32_t*>(us + kC * ldv + o) = lo;
                    } else {
                        u = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(vt + o));
                    }
                    split2(u.x * to_end[half], u.y * to_end[half], hi, lo);
                    *reinterpret_cast<uint32_t*>(ups + o) = hi;
                    *reinterpret_cast<uint32_t*>(ups + kC * ldv + o) = lo;
                }
            if (!DELTA) carriers_sync<kThreads / 2>();
        } else if (!RECORD) {
#pragma unroll 4
            for (int k = 0; k < ksteps; k++) {              // Q S0
                uint32_t f[4];
                ldsm4(f, qt + (warp * 16 + lda) * ld + k * 16 + ldb);
                times(acc, f, sh, k);
                times(low, f, sh + D16 * ldv, k);
            }
            join(acc, low);
            zero(low);
        }
        if (DELTA) __syncthreads();                         // U is there, and nobody reads the state any more
        if (carrier) {                                      // the state behind the chunk
            const float g_all = exp2_neg(1.4426950408889634f * end);
            each_state([&](float& x, bool, size_t) { x *= g_all; });
#pragma unroll
            for (int i = 0; i < MT; i++) {
                const int m0 = (warp + 4 * i) * 16;
                if (m0 >= D16) break;
                zero(low);
#pragma unroll
                for (int k = 0; k < kC / 16; k++) {
                    uint32_t f[4];
                    ldsm4t(f, kt + (k * 16 + (lane & 7) + ldb) * ld + m0 + ((lane >> 3) & 1) * 8);
                    times(S[i], f, ups, k);
                    times(low, f, ups + kC * ldv, k);
                }
                join(S[i], low);
            }
        } else if (!RECORD) {                               // outputs
#pragma unroll
            for (int j = 0; j < NT; j++)
#pragma unroll
                for (int e = 0; e < 4; e++) acc[j][e] *= dec[e >> 1] * rq[i0 + (e >> 1) * 8];
            for (int k = 0; k <= warp; k++) {
                uint32_t fh[4], fl[4];
                ldsm4(fh, pm + (warp * 16 + lda) * kLdC + k * 16 + ldb);
                ldsm4(fl, pm + kC * kLdC + (warp * 16 + lda) * kLdC + k * 16 + ldb);
                times(acc, fh, DELTA ? us : vt, k);
                times(low, fl, DELTA ? us : vt, k);
                if (DELTA) times(low, fh, us + kC * ldv, k);
            }
            join(acc, low);
#pragma unroll
            for (int half = 0; half < 2; half++) {
                const int i = i0 + half * 8;
                if (i >= n) continue;
                float* op = a.o + (row0 + (size_t)c * kC + i) * ((size_t)a.heads * a.vdim) + (size_t)h * a.vdim + v0;
#pragma unroll
                for (int j = 0; j < NT; j++) {
                    const int cc = n0 + j * 8 + 2 * tq;
                    if (cc < nv) *reinterpret_cast<float2*>(op + cc) = make_float2(acc[j][2 * half], acc[j][2 * half + 1]);
                }
            }
        }
        if ((!DELTA && !RECORD) || stages == 1) __syncthreads();   // nobody reads the state or the chunk any more
        if (carrier && !RECORD) save_state();
        if (requester && stages == 1 && c + 1 < c1) request(c + 1, 0);
    }
    if (!ok) {
        // copies may still be under way: they land before the shared memory goes away
        for (int s = 0; s < 2; s++) gemm::mbar_wait(gemm::smem_u32(&full[s]), 0, &never) || gemm::mbar_wait(gemm::smem_u32(&full[s]), 1, &never);
        if (lane == 0) atomicExch(ws.err, TLLM_ERR_TIMEOUT);
    }
    if (!carrier) return;
    float* last = RECORD ? rec + (size_t)seg * rec_size : st;
    if (RECORD || seg == nseg - 1) each_state([&](float& x, bool in, size_t o) { if (in) last[o] = x; });
}

size_t prepare_smem(bool delta, int dim)
{
    const int ld = ((dim + 15) & ~15) + 8;
    if (!delta) return (size_t)2 * kC * ld * 2;
    return (size_t)kC * ld * 2 + (size_t)(inverse_floats(ld) + kC * kLdA + (kC / 16 - 1) * 256) * 4;
}
size_t scan_smem(bool delta, int dim, int nv, int stages)
{
    const int d16 = (dim + 15) & ~15, ld = d16 + 8, ldv = nv + 8;
    const size_t stage = (size_t)(2 * kC * ld + chunk_mats(delta) * kC * kLdC + kC * ldv) * 2 + 4 * kC * 4;
    return stages * stage + (size_t)(2 * d16 * ldv + (delta ? 6 : 2) * kC * ldv) * 2;
}

constexpr size_t kSmemLimit = 220 * 1024;
constexpr int kChunkFrom = 48;                        // tokens from which chunks pay
constexpr int kChunkMaxDim = 256, kMaxSegments = 8, kSms = 148;

static_assert(kChunkFrom > kC / 2, "workspace bound");

bool chunked(int seq_len, int dim) { return seq_len >= kChunkFrom && dim <= kChunkMaxDim; }

template <bool DELTA, int NV, int MT>
int chunk_scan(const MatrixScanArgs<bf16>& a, const ChunkWs& ws, int nchunk, cudaStream_t stream)
{
    const int stages = scan_smem(DELTA, a.dim, NV, 2) <= kSmemLimit ? 2 : 1;
    const size_t smem = scan_smem(DELTA, a.dim, NV, stages);
    if (smem > kSmemLimit) return fail(TLLM_ERR_SHAPE, "matrix_scan: dim=%d", a.dim);
    const int slices = (a.vdim + NV - 1) / NV;
    int nseg = 1;
    if (!DELTA) {                                          // two chunks or more to a segment
        nseg = kSms / (slices * a.heads * a.g.n_seq);
        nseg = nseg > nchunk / 2 ? nchunk / 2 : nseg;
        nseg = nseg < 1 ? 1 : nseg > kMaxSegments ? kMaxSegments : nseg;
    }
    const int per = (nchunk + nseg - 1) / nseg;
    nseg = (nchunk + per - 1) / per;
    if (nseg > 1) {
        const auto kernel = chunk_scan_kernel<DELTA, NV, MT, !DELTA>;
        cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        const int st = launch_pdl("chunk_record", kernel, dim3(slices * (nseg - 1), a.heads, a.g.n_seq), dim3(kThreadsPerCol * NV), smem, stream, a, ws, nchunk,
                                  per, nseg, stages);
        if (st) return st;
    }
    const auto kernel = chunk_scan_kernel<DELTA, NV, MT, false>;
    cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    return launch_pdl("chunk_scan", kernel, dim3(slices * nseg, a.heads, a.g.n_seq), dim3(kThreadsPerCol * NV), smem, stream, a, ws, nchunk, per, nseg,
                      stages);
}

template <bool DELTA, int NV>
int chunk_scan_dim(const MatrixScanArgs<bf16>& a, const ChunkWs& ws, int nchunk, cudaStream_t stream)
{
    if (a.dim <= 64) return chunk_scan<DELTA, NV, 1>(a, ws, nchunk, stream);
    if (a.dim <= 128) return chunk_scan<DELTA, NV, 2>(a, ws, nchunk, stream);
    return chunk_scan<DELTA, NV, 4>(a, ws, nchunk, stream);
}

// bytes of the parts of ChunkWs, in order, for `chunks` chunks of all sequences
struct WsLayout {
    size_t kq, v, mats, vecs, rec;
    size_t total() const { return kq + v + mats + vecs + rec; }
};
WsLayout ws_layout(bool delta, size_t chunks, size_t segs, int heads, int kv_heads, int dim, int vdim, int nv)
{
    const size_t ld = ((dim + 15) & ~15) + 8, slices = (vdim + nv - 1) / nv, units = chunks * heads;
    WsLayout w;
    w.kq = chunks * kv_heads * 2 * kC * ld * sizeof(bf16);
    w.v = units * slices * kC * (nv + 8) * sizeof(bf16);
    w.mats = units * chunk_mats(delta) * kC * kLdC * sizeof(bf16);
    w.vecs = units * 4 * kC * sizeof(float);
    w.rec = delta ? 0 : segs * heads * vdim * dim * sizeof(float);
    return w;
}

template <bool DELTA>
int chunk_path(const MatrixScanArgs<bf16>& a, cudaStream_t stream)
{
    if (!a.ws) return fail(TLLM_ERR_NULL, "matrix_scan: no workspace");
    const int nchunk = chunks_of(a.g.seq_len);
    // narrow slices of the delta rule while they give more SMs one
    const bool narrow = DELTA && a.heads * a.g.n_seq * ((a.vdim + 31) / 32) * 2 <= kSms;
    const WsLayout l = ws_layout(DELTA, (size_t)a.g.n_seq * nchunk, 0, a.heads, a.kv_heads, a.dim, a.vdim, narrow ? 16 : 32);
    uint8_t* p = static_cast<uint8_t*>(a.ws);
    ChunkWs ws;
    ws.n_mats = (int)chunk_mats(DELTA);
    ws.nv = narrow ? 16 : 32;
    ws.kq = reinterpret_cast<bf16*>(p);
    ws.v = reinterpret_cast<bf16*>(p + l.kq);
    ws.mats = reinterpret_cast<bf16*>(p + l.kq + l.v);
    ws.vecs = reinterpret_cast<float*>(p + l.kq + l.v + l.mats);
    ws.rec = reinterpret_cast<float*>(p + l.total());
    ws.err = device_error_flag();
    if (!ws.err) return fail(TLLM_ERR_LAUNCH, "device scratch unavailable");
    const size_t smem = prepare_smem(DELTA, a.dim);
    cudaFuncSetAttribute(chunk_prepare_kernel<DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    int st = launch_pdl("chunk_prepare", chunk_prepare_kernel<DELTA>, dim3(nchunk, a.heads, a.g.n_seq), dim3(kChunkThreads), smem, stream, a, ws);
    if (st) return st;
    return narrow ? chunk_scan_dim<DELTA, 16>(a, ws, nchunk, stream) : chunk_scan_dim<DELTA, 32>(a, ws, nchunk, stream);
}
int chunk_any(const MatrixScanArgs<bf16>& a, cudaStream_t stream) { return a.delta ? chunk_path<true>(a, stream) : chunk_path<false>(a, stream); }
int chunk_any(const MatrixScanArgs<float>&, cudaStream_t) { return TLLM_ERR_SHAPE; }

template <typename T, bool DELTA>
__global__ void __launch_bounds__(kSeqThreads)
matrix_seq_kernel(const MatrixScanArgs<T> a, int lpc)
{
    extern __shared__ __align__(16) float smem[];
    pdl_launch_dependents();
    pdl_wait();
    matrix_seq<T, DELTA>(a, lpc, smem, blockIdx.x, blockIdx.y, blockIdx.z);
}

template <typename T, bool DELTA, bool NORM>
__global__ void __launch_bounds__(kSeqThreads)
matrix_one_kernel(const MatrixScanArgs<T> a, const GatedNormArgs<T> norm, int log_lpc)
{
    __shared__ float sh[kSeqThreads / 32 + kSeqMaxCluster];
    pdl_launch_dependents();
    pdl_wait();
    matrix_one<T, DELTA, NORM>(a, norm, log_lpc, sh, blockIdx.x, blockIdx.y, blockIdx.z);
}

template <typename T, bool DELTA>
int sequential(const MatrixScanArgs<T>& a, const GatedNormArgs<T>* norm, cudaStream_t stream)
{
    const SeqPlan p = seq_plan(a.dim, a.vdim);
    const dim3 grid(p.blocks, a.heads, a.g.n_seq);
    // one new token, a norm per head: the CTAs of a head share its sum of squares
    if (norm && a.g.seq_len == 1 && norm->groups == a.heads && p.blocks <= kSeqMaxCluster)
        return launch_pdl_cluster("matrix_one", matrix_one_kernel<T, DELTA, true>, p.blocks, grid, dim3(p.threads), 0, stream, a, *norm, p.log_lpc);
    const int st = a.g.seq_len == 1
                       ? launch_pdl("matrix_one", matrix_one_kernel<T, DELTA, false>, grid, dim3(p.threads), 0, stream, a, GatedNormArgs<T>(), p.log_lpc)
                       : launch_pdl("matrix_seq", matrix_seq_kernel<T, DELTA>, grid, dim3(p.threads), p.smem, stream, a, p.lpc);
    return st || !norm ? st : launch_gated_norm<T>(*norm, stream);
}

template <typename T>
__global__ void __launch_bounds__(kGnThreads)
gated_norm_kernel(const GatedNormArgs<T> a)
{
    __shared__ float sh[kGnWarps];
    pdl_launch_dependents();
    pdl_wait();
    gated_norm_row<T>(a, blockIdx.x, sh);
}

}  // namespace

size_t matrix_scan_workspace(bool bf16_path, bool delta, int rows, int heads, int kv_heads, int dim, int vdim)
{
    if (!bf16_path || !chunked(rows, dim)) return 0;
    const size_t chunks = (size_t)rows / (kC / 2) + 1;     // a sequence of 48 tokens or more: one chunk per 32 at most
    // records: a segment has two chunks or more
    const size_t segs = (size_t)rows / kC < kMaxSegments ? (size_t)rows / kC + 1 : kMaxSegments * ((size_t)rows / (kMaxSegments * kC) + 1);
    const size_t narrow = ws_layout(delta, chunks, segs, heads, kv_heads, dim, vdim, 16).total();
    const size_t wide = ws_layout(delta, chunks, segs, heads, kv_heads, dim, vdim, 32).total();
    return narrow > wide ? narrow : wide;
}

template <typename T>
int launch_matrix_scan(const MatrixScanArgs<T>& a, const GatedNormArgs<T>* norm, cudaStream_t stream)
{
    if (a.g.rows() == 0) return TLLM_OK;
    const int st = check_matrix_scan(a);
    if (st) return st;
    if (sizeof(T) == 2 && chunked(a.g.seq_len, a.dim)) {
        const int c = chunk_any(a, stream);
        return c || !norm ? c : launch_gated_norm<T>(*norm, stream);
    }
    return a.delta ? sequential<T, true>(a, norm, stream) : sequential<T, false>(a, norm, stream);
}

template <typename T>
int launch_gated_norm(const GatedNormArgs<T>& a, cudaStream_t stream)
{
    if (a.rows == 0) return TLLM_OK;
    if (a.n < 4 || a.n % 4 || a.groups < 1 || a.ld_gate % 4 || a.ld_out % 4) return fail(TLLM_ERR_SHAPE, "gated_norm: %d groups of %d", a.groups, a.n);
    return launch_pdl("gated_norm", gated_norm_kernel<T>, dim3(a.rows), dim3(kGnThreads), 0, stream, a);
}

#define TLLM_INSTANTIATE(T)                                                    \
    template int launch_matrix_scan<T>(const MatrixScanArgs<T>&, const GatedNormArgs<T>*, cudaStream_t); \
    template int launch_gated_norm<T>(const GatedNormArgs<T>&, cudaStream_t);
TLLM_INSTANTIATE(bf16)
TLLM_INSTANTIATE(float)
#undef TLLM_INSTANTIATE

}  // namespace tllm
