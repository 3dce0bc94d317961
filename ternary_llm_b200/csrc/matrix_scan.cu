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
#include "mixers.cuh"
#include "mma_sync.cuh"

namespace tllm {

namespace {

constexpr float kUnitEps = 1e-6f;     // under the root of the unit vectors

__device__ __forceinline__ float log_decay(float a, float dt_bias, float neg_a) { return neg_a * softplus_f(a + dt_bias); }

// ---------------------------------------------------------------------------
// Token by token
// ---------------------------------------------------------------------------
constexpr int kSeqThreads = 256, kSeqStates = 16, kSeqTokens = 8;   // entries of a column per lane; tokens staged together

// A column of S is spread over `lpc` lanes in pieces of four entries; a CTA serves blockDim / lpc
// columns of one head.
template <typename T, bool DELTA>
__global__ void __launch_bounds__(kSeqThreads)
matrix_seq_kernel(const MatrixScanArgs<T> a, int lpc)
{
    extern __shared__ __align__(16) float smem[];
    constexpr int NP = kSeqStates / 4;
    const int cols = blockDim.x / lpc, D = a.dim, D4 = D >> 2;
    float* ks = smem;                                   // [tokens][D]
    float* qs = ks + kSeqTokens * D;
    float* vs = qs + kSeqTokens * D;                    // [tokens][cols]
    float* gs = vs + kSeqTokens * cols;                 // decay, step size
    float* bs = gs + kSeqTokens;
    pdl_launch_dependents();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, warps = blockDim.x >> 5;
    const int cl = tid / lpc, l = tid - cl * lpc, c0 = blockIdx.x * cols, c = c0 + cl, h = blockIdx.y, b = blockIdx.z;
    const int kh = h / (a.heads / a.kv_heads);
    const bool live = c < a.vdim;
    pdl_wait();
    const bool fresh = (a.g.pos_dev ? *a.g.pos_dev : a.g.start_pos) == 0;
    float4* st = reinterpret_cast<float4*>(a.state + (size_t)(a.g.first_slot + b) * a.slot_stride + ((size_t)h * a.vdim + (live ? c : 0)) * D);
    float4 S[NP];
#pragma unroll
    for (int u = 0; u < NP; u++) {
        const int p = l + u * lpc;
        S[u] = (live && !fresh && p < D4) ? st[p] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const int n = a.g.seq_len;
    const size_t row0 = (size_t)b * n;
    for (int t0 = 0; t0 < n; t0 += kSeqTokens) {
        const int nt = min(kSeqTokens, n - t0);
        __syncthreads();
        // a warp per vector: keys, queries, values of the staged tokens
        for (int i = warp; i < 3 * nt; i += warps) {
            const int t = i / 3, what = i - 3 * t;
            const size_t row = row0 + t0 + t;
            if (what == 2) {
                const T* v = a.v + row * a.ld + (size_t)h * a.vdim + c0;
                for (int j = lane; j < cols; j += 32) vs[t * cols + j] = c0 + j < a.vdim ? to_f<T>(v[j]) : 0.f;
                if (lane == 0) {
                    if (DELTA) {
                        const float lg = log_decay(a.a[row * a.ld_ab + h], a.dt_bias[h], a.neg_a[h]);
                        gs[t] = decay_exp(lg, expf(lg));
                        bs[t] = sigmoid_f(a.b[row * a.ld_ab + h]);
                    } else {
                        gs[t] = a.decay[h];
                    }
                }
                continue;
            }
            const T* x = (what ? a.q : a.k) + row * a.ld + (size_t)kh * D;
            float* dst = (what ? qs : ks) + t * D;
            float f = 1.f;
            if (DELTA) {
                float ss = 0.f;
                for (int j = lane; j < D; j += 32) {
                    const float v = to_f<T>(x[j]);
                    ss += v * v;
                }
                f = 1.f / sqrtf(warp_sum(ss) + kUnitEps);
                if (what) f *= a.q_scale;
            }
            for (int j = lane; j < D; j += 32) dst[j] = to_f<T>(x[j]) * f;
        }
        __syncthreads();
        for (int t = 0; t < nt; t++) {
            const float g = gs[t];
            const float4 *kp = reinterpret_cast<const float4*>(ks + t * D), *qp = reinterpret_cast<const float4*>(qs + t * D);
            float4 k[NP];
#pragma unroll
            for (int u = 0; u < NP; u++) k[u] = l + u * lpc < D4 ? kp[l + u * lpc] : make_float4(0.f, 0.f, 0.f, 0.f);
            float add = vs[t * cols + cl];
            if (DELTA) {
                float p = 0.f;
#pragma unroll
                for (int u = 0; u < NP; u++) {
                    S[u].x *= g;
                    S[u].y *= g;
                    S[u].z *= g;
                    S[u].w *= g;
                    p = fmaf(S[u].x, k[u].x, fmaf(S[u].y, k[u].y, fmaf(S[u].z, k[u].z, fmaf(S[u].w, k[u].w, p))));
                }
                for (int o = lpc >> 1; o > 0; o >>= 1) p += __shfl_xor_sync(0xffffffffu, p, o);
                add = bs[t] * (add - p);
            }
            float o = 0.f;
#pragma unroll
            for (int u = 0; u < NP; u++) {
                const float d = DELTA ? 1.f : g;
                S[u].x = fmaf(k[u].x, add, d * S[u].x);
                S[u].y = fmaf(k[u].y, add, d * S[u].y);
                S[u].z = fmaf(k[u].z, add, d * S[u].z);
                S[u].w = fmaf(k[u].w, add, d * S[u].w);
                if (l + u * lpc < D4) {
                    const float4 q = qp[l + u * lpc];
                    o = fmaf(S[u].x, q.x, fmaf(S[u].y, q.y, fmaf(S[u].z, q.z, fmaf(S[u].w, q.w, o))));
                }
            }
            for (int s = lpc >> 1; s > 0; s >>= 1) o += __shfl_xor_sync(0xffffffffu, o, s);
            if (live && l == 0) a.o[(row0 + t0 + t) * ((size_t)a.heads * a.vdim) + (size_t)h * a.vdim + c] = o;
        }
    }
    if (live) {
#pragma unroll
        for (int u = 0; u < NP; u++)
            if (l + u * lpc < D4) st[l + u * lpc] = S[u];
    }
}

// ---------------------------------------------------------------------------
// Chunks
// ---------------------------------------------------------------------------
constexpr int kC = 64, kChunkThreads = 128;
constexpr int kLdC = kC + 8;                       // row stride of a [64][64] tile in shared memory

// per (sequence, chunk, head): matrices [64][64], BF16 high and low parts -- P, then with the delta
// rule the inverse -- and four vectors of 64 floats (log of the running decay, step size, 1/|k|,
// q_scale/|q|)
struct ChunkWs {
    bf16* mats;
    float* vecs;
    int n_mats;
};
__host__ __device__ inline size_t chunk_mats(bool delta) { return delta ? 4 : 2; }
inline int chunks_of(int n) { return (n + kC - 1) / kC; }

template <bool DELTA>
__global__ void __launch_bounds__(kChunkThreads)
chunk_prepare_kernel(const MatrixScanArgs<bf16> a, ChunkWs ws)
{
    extern __shared__ __align__(16) uint8_t smem_raw[];
    const int D = a.dim, ld = ((D + 15) & ~15) + 8, ksteps = (D + 15) / 16;
    bf16* ks = reinterpret_cast<bf16*>(smem_raw);          // [64][ld]
    bf16* qs = ks + kC * ld;
    float* A = reinterpret_cast<float*>(qs + kC * ld);     // [64][64] (delta)
    __shared__ float logg[kC], beta[kC], rk[kC], rq[kC];
    pdl_launch_dependents();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int chunk = blockIdx.x, h = blockIdx.y, b = blockIdx.z, kh = h / (a.heads / a.kv_heads);
    const int n = min(kC, a.g.seq_len - chunk * kC);
    const size_t row0 = (size_t)b * a.g.seq_len + (size_t)chunk * kC;
    const size_t unit = ((size_t)b * gridDim.x + chunk) * a.heads + h;
    bf16* mats = ws.mats + unit * ws.n_mats * kC * kC;
    pdl_wait();
    {
        const int pieces = D / 8, per = ld / 8;
        for (int i = tid; i < kC * per; i += kChunkThreads) {
            const int r = i / per, c = i - r * per;
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
    cp_wait<0>();
    __syncthreads();
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
                *reinterpret_cast<uint32_t*>(mats + i * kC + c) = hi;
                *reinterpret_cast<uint32_t*>(mats + kC * kC + i * kC + c) = lo;
            }
    };
    if (!DELTA) {
        write_p(warp * 16);
        return;
    }
    {
        float s[8][4];
        gram(ks, warp * 16, s);
#pragma unroll
        for (int j = 0; j < 8; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int i = warp * 16 + (lane >> 2) + (e >> 1) * 8, c = j * 8 + 2 * (lane & 3) + (e & 1);
                A[i * kC + c] = c < i ? beta[i] * weight(i, c) * rk[i] * rk[c] * s[j][e] : 0.f;
            }
    }
    __syncthreads();
    if (warp >= 2) {
        write_p((warp - 2) * 16);
        write_p((5 - warp) * 16);                           // warps 2, 3: rows 0, 48 and 16, 32
        return;
    }
    // forward substitution, a column of the inverse per thread
    float x[kC];
#pragma unroll
    for (int i = 0; i < kC; i++) {
        float s0 = i == tid ? 1.f : 0.f, s1 = 0.f;
#pragma unroll
        for (int j = 0; j < i; j += 4) {
            const float4 r = *reinterpret_cast<const float4*>(A + i * kC + j);   // zeros from the diagonal on
            s0 = fmaf(-r.x, x[j], s0);
            if (j + 1 < i) s1 = fmaf(-r.y, x[j + 1], s1);
            if (j + 2 < i) s0 = fmaf(-r.z, x[j + 2], s0);
            if (j + 3 < i) s1 = fmaf(-r.w, x[j + 3], s1);
        }
        x[i] = s0 + s1;
        const bf16 hi = __float2bfloat16_rn(x[i]);
        mats[2 * kC * kC + i * kC + tid] = hi;
        mats[3 * kC * kC + i * kC + tid] = __float2bfloat16_rn(x[i] - __bfloat162float(hi));
    }
}

// NV columns of the state per CTA, MT tiles of 16 state rows per warp; `stages` chunks in flight
template <bool DELTA, int NV, int MT>
__global__ void __launch_bounds__(kChunkThreads)
chunk_scan_kernel(const MatrixScanArgs<bf16> a, ChunkWs ws, int nchunk, int stages)
{
    extern __shared__ __align__(16) uint8_t smem_raw[];
    constexpr int ldv = NV + 8, NT = NV / 8, MATS = DELTA ? 4 : 2;
    const int D = a.dim, D16 = (D + 15) & ~15, ld = D16 + 8, ksteps = D16 / 16;
    const int tile = 2 * kC * ld + MATS * kC * kLdC + kC * ldv;               // bf16 of a stage, then 4 * 64 floats
    const size_t stage_bytes = (size_t)tile * 2 + 4 * kC * sizeof(float);
    bf16* sh = reinterpret_cast<bf16*>(smem_raw + stages * stage_bytes);       // state [D16][ldv], high and low
    bf16* rs = sh + 2 * D16 * ldv;                                             // right-hand side [64][ldv], high and low
    bf16* us = rs + (DELTA ? 2 * kC * ldv : 0);                                // U
    bf16* ups = us + (DELTA ? 2 * kC * ldv : 0);                               // U times its decay to the end
    pdl_launch_dependents();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, tq = lane & 3;
    const int v0 = blockIdx.x * NV, h = blockIdx.y, b = blockIdx.z, kh = h / (a.heads / a.kv_heads);
    const int nv = min(NV, a.vdim - v0);
    const size_t row0 = (size_t)b * a.g.seq_len;
    pdl_wait();
    const bool fresh = (a.g.pos_dev ? *a.g.pos_dev : a.g.start_pos) == 0;
    float* st = a.state + (size_t)(a.g.first_slot + b) * a.slot_stride + ((size_t)h * a.vdim + v0) * D;

    auto request = [&](int c, int stage) {
        bf16* p = reinterpret_cast<bf16*>(smem_raw + stage * stage_bytes);
        const int n = min(kC, a.g.seq_len - c * kC), per = ld / 8, pieces = D / 8;
        const size_t r0 = row0 + (size_t)c * kC, unit = ((size_t)b * nchunk + c) * a.heads + h;
        for (int i = tid; i < kC * per; i += kChunkThreads) {
            const int r = i / per, cc = i - r * per;
            const bool v = r < n && cc < pieces;
            const size_t o = (r0 + (v ? r : 0)) * a.ld + (size_t)kh * D + (v ? cc * 8 : 0);
            cp16(p + r * ld + cc * 8, a.k + o, v);
            cp16(p + kC * ld + r * ld + cc * 8, a.q + o, v);
        }
        p += 2 * kC * ld;
        const bf16* m = ws.mats + unit * MATS * kC * kC;
        for (int i = tid; i < MATS * kC * (kC / 8); i += kChunkThreads)
            cp16(p + (i >> 3) * kLdC + (i & 7) * 8, m + (size_t)i * 8, true);
        p += MATS * kC * kLdC;
        for (int i = tid; i < kC * (NV / 8); i += kChunkThreads) {
            const int r = i / (NV / 8), cc = (i - r * (NV / 8)) * 8;
            const bool v = r < n && cc < nv;
            cp16(p + r * ldv + cc, a.v + (r0 + (v ? r : 0)) * a.ld + (size_t)h * a.vdim + v0 + (v ? cc : 0), v);
        }
        p += kC * ldv;
        const float* vec = ws.vecs + unit * 4 * kC;
        for (int i = tid; i < kC; i += kChunkThreads) cp16(p + 8 * i, reinterpret_cast<const bf16*>(vec + 4 * i), true);
        cp_commit();
    };
    request(0, 0);

    float S[MT][NT][4];
    auto each_state = [&](auto&& f) {                       // (tile, column tile, element, row, column)
#pragma unroll
        for (int i = 0; i < MT; i++)
#pragma unroll
            for (int j = 0; j < NT; j++)
#pragma unroll
                for (int e = 0; e < 4; e++) f(i, j, e, (warp + 4 * i) * 16 + gq + (e >> 1) * 8, j * 8 + 2 * tq + (e & 1));
    };
    each_state([&](int i, int j, int e, int r, int c) { S[i][j][e] = (!fresh && r < D && c < nv) ? st[(size_t)c * D + r] : 0.f; });
    const int lda = lane & 15, ldb = (lane >> 4) * 8;
    const int i0 = warp * 16 + gq;                          // this lane's rows i0 and i0 + 8 of a chunk

    for (int c = 0; c < nchunk; c++) {
        const int stage = stages == 2 ? c & 1 : 0, n = min(kC, a.g.seq_len - c * kC);
        const bf16* kt = reinterpret_cast<const bf16*>(smem_raw + stage * stage_bytes);
        const bf16 *qt = kt + kC * ld, *pm = qt + kC * ld, *tm = pm + 2 * kC * kLdC, *vt = pm + MATS * kC * kLdC;
        const float* logg = reinterpret_cast<const float*>(vt + kC * ldv);
        const float *beta = logg + kC, *rk = beta + kC, *rq = rk + kC;
        // the state as two BF16 matrices
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
                    const int o = (r + half * 8) * ldv + j * 8 + 2 * tq;
                    *reinterpret_cast<uint32_t*>(sh + o) = hi;
                    *reinterpret_cast<uint32_t*>(sh + D16 * ldv + o) = lo;
                }
        }
        cp_wait<0>();
        __syncthreads();
        if (stages == 2 && c + 1 < nchunk) request(c + 1, stage ^ 1);
        // K S0 and Q S0, 16 rows per warp
        float ksum[NT][4], qsum[NT][4];
#pragma unroll
        for (int j = 0; j < NT; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) ksum[j][e] = qsum[j][e] = 0.f;
#pragma unroll 2
        for (int k = 0; k < ksteps; k++) {
            uint32_t fk[4], fq[4];
            if (DELTA) ldsm4(fk, kt + (warp * 16 + lda) * ld + k * 16 + ldb);
            ldsm4(fq, qt + (warp * 16 + lda) * ld + k * 16 + ldb);
#pragma unroll
            for (int part = 0; part < 2; part++)
#pragma unroll
                for (int j = 0; j < NT; j += 2) {
                    uint32_t fb[4];
                    ldsm4t(fb, sh + part * D16 * ldv + (k * 16 + lda) * ldv + j * 8 + ldb);
                    if (DELTA) {
                        mma16816(ksum[j], fk, fb[0], fb[1]);
                        mma16816(ksum[j + 1], fk, fb[2], fb[3]);
                    }
                    mma16816(qsum[j], fq, fb[0], fb[1]);
                    mma16816(qsum[j + 1], fq, fb[2], fb[3]);
                }
        }
        const float end = logg[n - 1];
        float dec[2], to_end[2];
#pragma unroll
        for (int half = 0; half < 2; half++) {
            const int i = i0 + half * 8;
            dec[half] = exp2_neg(1.4426950408889634f * logg[i]);
            to_end[half] = i < n ? exp2_neg(1.4426950408889634f * (end - logg[i])) * rk[i] : 0.f;
        }
        if (DELTA) {
#pragma unroll
            for (int j = 0; j < NT; j++)
#pragma unroll
                for (int half = 0; half < 2; half++) {
                    const int i = i0 + half * 8, o = i * ldv + j * 8 + 2 * tq;
                    const float f = dec[half] * rk[i], be = beta[i];
                    const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(vt + o));
                    uint32_t hi, lo;
                    split2(be * (v.x - f * ksum[j][2 * half]), be * (v.y - f * ksum[j][2 * half + 1]), hi, lo);
                    *reinterpret_cast<uint32_t*>(rs + o) = hi;
                    *reinterpret_cast<uint32_t*>(rs + kC * ldv + o) = lo;
                }
            __syncthreads();
            float u[NT][4];
#pragma unroll
            for (int j = 0; j < NT; j++)
#pragma unroll
                for (int e = 0; e < 4; e++) u[j][e] = 0.f;
            for (int k = 0; k <= warp; k++) {              // triangular
                uint32_t fh[4], fl[4];
                ldsm4(fh, tm + (warp * 16 + lda) * kLdC + k * 16 + ldb);
                ldsm4(fl, tm + kC * kLdC + (warp * 16 + lda) * kLdC + k * 16 + ldb);
#pragma unroll
                for (int j = 0; j < NT; j += 2) {
                    uint32_t fb[4], fc[4];
                    ldsm4t(fb, rs + (k * 16 + lda) * ldv + j * 8 + ldb);
                    ldsm4t(fc, rs + kC * ldv + (k * 16 + lda) * ldv + j * 8 + ldb);
                    mma16816(u[j], fh, fb[0], fb[1]);
                    mma16816(u[j + 1], fh, fb[2], fb[3]);
                    mma16816(u[j], fl, fb[0], fb[1]);
                    mma16816(u[j + 1], fl, fb[2], fb[3]);
                    mma16816(u[j], fh, fc[0], fc[1]);
                    mma16816(u[j + 1], fh, fc[2], fc[3]);
                }
            }
#pragma unroll
            for (int j = 0; j < NT; j++)
#pragma unroll
                for (int half = 0; half < 2; half++) {
                    const int o = (i0 + half * 8) * ldv + j * 8 + 2 * tq;
                    uint32_t hi, lo;
                    split2(u[j][2 * half], u[j][2 * half + 1], hi, lo);
                    *reinterpret_cast<uint32_t*>(us + o) = hi;
                    *reinterpret_cast<uint32_t*>(us + kC * ldv + o) = lo;
                    split2(u[j][2 * half] * to_end[half], u[j][2 * half + 1] * to_end[half], hi, lo);
                    *reinterpret_cast<uint32_t*>(ups + o) = hi;
                    *reinterpret_cast<uint32_t*>(ups + kC * ldv + o) = lo;
                }
        } else {
#pragma unroll
            for (int j = 0; j < NT; j++)
#pragma unroll
                for (int half = 0; half < 2; half++) {
                    const int o = (i0 + half * 8) * ldv + j * 8 + 2 * tq;
                    const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(vt + o));
                    uint32_t hi, lo;
                    split2(v.x * to_end[half], v.y * to_end[half], hi, lo);
                    *reinterpret_cast<uint32_t*>(ups + o) = hi;
                    *reinterpret_cast<uint32_t*>(ups + kC * ldv + o) = lo;
                }
        }
        __syncthreads();
        // outputs
#pragma unroll
        for (int j = 0; j < NT; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) qsum[j][e] *= dec[e >> 1] * rq[i0 + (e >> 1) * 8];
        const bf16* ub = DELTA ? us : vt;
        for (int k = 0; k <= warp; k++) {
            uint32_t fh[4], fl[4];
            ldsm4(fh, pm + (warp * 16 + lda) * kLdC + k * 16 + ldb);
            ldsm4(fl, pm + kC * kLdC + (warp * 16 + lda) * kLdC + k * 16 + ldb);
#pragma unroll
            for (int j = 0; j < NT; j += 2) {
                uint32_t fb[4];
                ldsm4t(fb, ub + (k * 16 + lda) * ldv + j * 8 + ldb);
                mma16816(qsum[j], fh, fb[0], fb[1]);
                mma16816(qsum[j + 1], fh, fb[2], fb[3]);
                mma16816(qsum[j], fl, fb[0], fb[1]);
                mma16816(qsum[j + 1], fl, fb[2], fb[3]);
                if (DELTA) {
                    ldsm4t(fb, us + kC * ldv + (k * 16 + lda) * ldv + j * 8 + ldb);
                    mma16816(qsum[j], fh, fb[0], fb[1]);
                    mma16816(qsum[j + 1], fh, fb[2], fb[3]);
                }
            }
        }
#pragma unroll
        for (int half = 0; half < 2; half++) {
            const int i = i0 + half * 8;
            if (i >= n) continue;
            float* op = a.o + (row0 + (size_t)c * kC + i) * ((size_t)a.heads * a.vdim) + (size_t)h * a.vdim + v0;
#pragma unroll
            for (int j = 0; j < NT; j++) {
                const int cc = j * 8 + 2 * tq;
                if (cc < nv) *reinterpret_cast<float2*>(op + cc) = make_float2(qsum[j][2 * half], qsum[j][2 * half + 1]);
            }
        }
        // the state behind the chunk
        const float g_all = exp2_neg(1.4426950408889634f * end);
        each_state([&](int i, int j, int e, int, int) { S[i][j][e] *= g_all; });
#pragma unroll
        for (int i = 0; i < MT; i++) {
            const int m0 = (warp + 4 * i) * 16;
            if (m0 >= D16) break;
#pragma unroll
            for (int k = 0; k < kC / 16; k++) {
                uint32_t fa[4];
                ldsm4t(fa, kt + (k * 16 + (lane & 7) + ldb) * ld + m0 + ((lane >> 3) & 1) * 8);
#pragma unroll
                for (int part = 0; part < 2; part++)
#pragma unroll
                    for (int j = 0; j < NT; j += 2) {
                        uint32_t fb[4];
                        ldsm4t(fb, ups + part * kC * ldv + (k * 16 + lda) * ldv + j * 8 + ldb);
                        mma16816(S[i][j], fa, fb[0], fb[1]);
                        mma16816(S[i][j + 1], fa, fb[2], fb[3]);
                    }
            }
        }
        if (stages == 1) {
            __syncthreads();
            if (c + 1 < nchunk) request(c + 1, 0);
        }
    }
    each_state([&](int i, int j, int e, int r, int c) {
        if (r < D && c < nv) st[(size_t)c * D + r] = S[i][j][e];
    });
}

size_t prepare_smem(bool delta, int dim)
{
    return (size_t)2 * kC * (((dim + 15) & ~15) + 8) * 2 + (delta ? (size_t)kC * kC * 4 : 0);
}
size_t scan_smem(bool delta, int dim, int nv, int stages)
{
    const int d16 = (dim + 15) & ~15, ld = d16 + 8, ldv = nv + 8;
    const size_t stage = (size_t)(2 * kC * ld + chunk_mats(delta) * kC * kLdC + kC * ldv) * 2 + 4 * kC * 4;
    return stages * stage + (size_t)(2 * d16 * ldv + (delta ? 6 : 2) * kC * ldv) * 2;
}

constexpr size_t kSmemLimit = 220 * 1024;
constexpr int kChunkNv = 32, kChunkFrom = 48;         // columns per CTA; tokens from which chunks pay
constexpr int kChunkMaxDim = 256;

static_assert(kChunkFrom > kC / 2, "workspace bound");

bool chunked(int seq_len, int dim) { return seq_len >= kChunkFrom && dim <= kChunkMaxDim; }

template <bool DELTA, int MT>
int chunk_scan(const MatrixScanArgs<bf16>& a, const ChunkWs& ws, int nchunk, cudaStream_t stream)
{
    const int stages = scan_smem(DELTA, a.dim, kChunkNv, 2) <= kSmemLimit ? 2 : 1;
    const size_t smem = scan_smem(DELTA, a.dim, kChunkNv, stages);
    const auto kernel = chunk_scan_kernel<DELTA, kChunkNv, MT>;
    cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    return launch_pdl("chunk_scan", kernel, dim3((a.vdim + kChunkNv - 1) / kChunkNv, a.heads, a.g.n_seq), dim3(kChunkThreads), smem, stream, a, ws,
                      nchunk, stages);
}

template <bool DELTA>
int chunk_path(const MatrixScanArgs<bf16>& a, cudaStream_t stream)
{
    if (!a.ws) return fail(TLLM_ERR_NULL, "matrix_scan: no workspace");
    const int nchunk = chunks_of(a.g.seq_len);
    const size_t units = (size_t)a.g.n_seq * nchunk * a.heads;
    ChunkWs ws;
    ws.n_mats = (int)chunk_mats(DELTA);
    ws.mats = static_cast<bf16*>(a.ws);
    ws.vecs = reinterpret_cast<float*>(ws.mats + units * ws.n_mats * kC * kC);
    const size_t smem = prepare_smem(DELTA, a.dim);
    cudaFuncSetAttribute(chunk_prepare_kernel<DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    int st = launch_pdl("chunk_prepare", chunk_prepare_kernel<DELTA>, dim3(nchunk, a.heads, a.g.n_seq), dim3(kChunkThreads), smem, stream, a, ws);
    if (st) return st;
    if (a.dim <= 64) return chunk_scan<DELTA, 1>(a, ws, nchunk, stream);
    if (a.dim <= 128) return chunk_scan<DELTA, 2>(a, ws, nchunk, stream);
    return chunk_scan<DELTA, 4>(a, ws, nchunk, stream);
}
int chunk_any(const MatrixScanArgs<bf16>& a, cudaStream_t stream) { return a.delta ? chunk_path<true>(a, stream) : chunk_path<false>(a, stream); }
int chunk_any(const MatrixScanArgs<float>&, cudaStream_t) { return TLLM_ERR_SHAPE; }

template <typename T, bool DELTA>
int sequential(const MatrixScanArgs<T>& a, cudaStream_t stream)
{
    int lpc = 1;
    while (lpc * kSeqStates < a.dim) lpc *= 2;
    int threads = kSeqThreads;
    while (threads > 32 && threads / 2 / lpc >= a.vdim) threads /= 2;
    const int cols = threads / lpc;
    const size_t smem = (size_t)kSeqTokens * (2 * a.dim + cols + 2) * sizeof(float);
    return launch_pdl("matrix_seq", matrix_seq_kernel<T, DELTA>, dim3((a.vdim + cols - 1) / cols, a.heads, a.g.n_seq), dim3(threads), smem, stream, a,
                      lpc);
}

// ---------------------------------------------------------------------------
// Gated norm
// ---------------------------------------------------------------------------
constexpr int kGnThreads = 256, kGnWarps = kGnThreads / 32;

__device__ __forceinline__ void put4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void put4(bf16* p, float4 v)
{
    const __nv_bfloat162 x = __floats2bfloat162_rn(v.x, v.y), y = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&x), *reinterpret_cast<const uint32_t*>(&y));
}
__device__ __forceinline__ float4 get4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 get4(const bf16* p)
{
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16),
                       __uint_as_float(v.y & 0xffff0000u));
}

// CTA per row; a warp per group, or the whole CTA when the row is one group
template <typename T>
__global__ void __launch_bounds__(kGnThreads)
gated_norm_kernel(const GatedNormArgs<T> a)
{
    __shared__ float sh[kGnWarps];
    pdl_launch_dependents();
    const int row = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const bool whole = a.groups == 1;
    const int step = whole ? kGnThreads : 32, i0 = whole ? tid : lane, n4 = a.n >> 2;
    pdl_wait();
    for (int g = whole ? 0 : warp; g < a.groups; g += whole ? 1 : kGnWarps) {
        const float* o = a.o + ((size_t)row * a.groups + g) * a.n;
        const T* gate = a.gate + (size_t)row * a.ld_gate + (size_t)g * a.n;
        T* out = a.out + (size_t)row * a.ld_out + (size_t)g * a.n;
        float ss = 0.f;
        for (int i = i0; i < n4; i += step) {
            const float4 v = get4(o + 4 * i);
            ss += (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w);
        }
        ss = warp_sum(ss);
        if (whole) {
            if (lane == 0) sh[warp] = ss;
            __syncthreads();
            ss = 0.f;
#pragma unroll
            for (int i = 0; i < kGnWarps; i++) ss += sh[i];
        }
        const float r = a.out_scale / sqrtf(ss / (float)a.n_true + a.eps);
        for (int i = i0; i < n4; i += step) {
            const float4 v = get4(o + 4 * i), w = get4(a.w + 4 * i), z = get4(gate + 4 * i);
            float t[4] = {z.x, z.y, z.z, z.w};
            apply_act_n<4>(a.act, t);
            put4(out + 4 * i, make_float4(v.x * r * w.x * t[0], v.y * r * w.y * t[1], v.z * r * w.z * t[2], v.w * r * w.w * t[3]));
        }
    }
}

}  // namespace

size_t matrix_scan_workspace(bool bf16_path, bool delta, int rows, int heads, int dim)
{
    if (!bf16_path || !chunked(rows, dim)) return 0;
    const size_t units = ((size_t)rows / (kC / 2) + 1) * heads;      // a sequence of 48 tokens or more: one chunk per 32 at most
    return units * (chunk_mats(delta) * kC * kC * sizeof(bf16) + 4 * kC * sizeof(float));
}

template <typename T>
int launch_matrix_scan(const MatrixScanArgs<T>& a, cudaStream_t stream)
{
    if (a.g.rows() == 0) return TLLM_OK;
    if (a.heads < 1 || a.kv_heads < 1 || a.heads % a.kv_heads || a.dim < 8 || a.dim % 8 || a.dim > 512 || a.vdim < 8 || a.vdim % 8 || a.ld % 8 ||
        (a.delta ? !a.a || !a.b || !a.neg_a || !a.dt_bias : !a.decay))
        return fail(TLLM_ERR_SHAPE, "matrix_scan: heads=%d/%d dim=%d (8..512) vdim=%d ld=%d", a.heads, a.kv_heads, a.dim, a.vdim, a.ld);
    if (sizeof(T) == 2 && chunked(a.g.seq_len, a.dim)) return chunk_any(a, stream);
    return a.delta ? sequential<T, true>(a, stream) : sequential<T, false>(a, stream);
}

template <typename T>
int launch_gated_norm(const GatedNormArgs<T>& a, cudaStream_t stream)
{
    if (a.rows == 0) return TLLM_OK;
    if (a.n < 4 || a.n % 4 || a.groups < 1 || a.ld_gate % 4 || a.ld_out % 4) return fail(TLLM_ERR_SHAPE, "gated_norm: %d groups of %d", a.groups, a.n);
    return launch_pdl("gated_norm", gated_norm_kernel<T>, dim3(a.rows), dim3(kGnThreads), 0, stream, a);
}

#define TLLM_INSTANTIATE(T)                                                    \
    template int launch_matrix_scan<T>(const MatrixScanArgs<T>&, cudaStream_t); \
    template int launch_gated_norm<T>(const GatedNormArgs<T>&, cudaStream_t);
TLLM_INSTANTIATE(bf16)
TLLM_INSTANTIATE(float)
#undef TLLM_INSTANTIATE

}  // namespace tllm
