// Latent attention: keys and values of all heads are linear functions of one cached latent
// vector per position; a rotated key part shared by the heads is cached beside it.  Softmax in
// FP32, with an optional learned term per head in the denominator.
//
// Two forms of the same product:
//   absorbed -- queries are taken into latent space (W_uk applied to the query), every head
//     attends to the same cache rows, which serve as keys AND values, and W_uv is applied to
//     the result.  The cache row is read once for 16 (token, head) pairs, which is what a decode
//     step wants: the positions are split over CTAs, partial results are merged afterwards.
//   expanded -- keys and values of the whole context are computed once and a tile of 64 queries
//     of one head walks over them: fewer operations per (query, key) pair, for prompts.
// The BF16 kernels run on mma.sync with FP32 scores; the softmax weights enter the second
// product as the sum of two BF16 numbers (high part and remainder), so they keep 16 bits.
// The exact 32-bit mode uses the plain kernel below, which also takes latents wider than the
// tensor-core form has registers for.
#include <cfloat>

#include "launch.cuh"
#include "mixers.cuh"
#include "mma_sync.cuh"

namespace tllm {

namespace {

constexpr float kLog2e = 1.4426950408889634f;

// ---------------------------------------------------------------------------
// Latent norm, rotations, cache append
// ---------------------------------------------------------------------------
constexpr int kPrepThreads = 256;

template <typename T>
__global__ void __launch_bounds__(kPrepThreads)
latent_prep_kernel(const LatentArgs<T> a, T* __restrict__ q_abs)
{
    __shared__ float sh[kPrepThreads / 32];
    pdl_launch_dependents();
    const int row = blockIdx.x, b = row / a.g.seq_len, t = row - b * a.g.seq_len;
    const int tid = threadIdx.x, half_dims = a.rot_dims >> 1;
    pdl_wait();
    const int pos = (a.g.pos_dev ? *a.g.pos_dev : a.g.start_pos) + t;
    if (pos >= a.max_seq) return;
    T* proj = a.proj + (size_t)row * a.ld;
    T* cache = a.cache + (size_t)(a.g.first_slot + b) * a.slot_stride + (size_t)pos * (a.rank + a.rot);
    const float2* cs = a.rope + (size_t)pos * half_dims;

    if (blockIdx.y == 0) {       // the latent
        float ss = 0.f;
        for (int i = tid; i < a.rank; i += kPrepThreads) {
            const float v = to_f<T>(proj[a.kv_off + i]);
            ss += v * v;
        }
        ss = warp_sum(ss);
        if ((tid & 31) == 0) sh[tid >> 5] = ss;
        __syncthreads();
        ss = 0.f;
#pragma unroll
        for (int i = 0; i < kPrepThreads / 32; i++) ss += sh[i];
        const float rinv = 1.0f / sqrtf(ss / (float)a.rank_true + a.eps);
        for (int i = tid; i < a.rank; i += kPrepThreads) cache[i] = from_f<T>(to_f<T>(proj[a.kv_off + i]) * rinv * a.kv_norm[i]);
        return;
    }

    // rotated parts: head -1 is the shared key part
    const int per = a.rot - half_dims;                      // half_dims pairs, then the entries that pass
    const int dk = a.rank + a.rot;
#pragma unroll 2
    for (int i = tid; i < (a.heads + 1) * per; i += kPrepThreads) {
        const int h = i / per - 1, e = i - (h + 1) * per;
        const T* src = (h < 0) ? proj + a.kv_off + a.rank : proj + a.q_off + (size_t)h * (a.dim + a.rot) + a.dim;
        T* dst = (h < 0) ? cache + a.rank : const_cast<T*>(src);
        T* dst2 = (h >= 0 && q_abs) ? q_abs + ((size_t)row * a.heads + h) * dk + a.rank : nullptr;
        if (e < half_dims) {
            const float u = to_f<T>(src[e]), v = to_f<T>(src[e + half_dims]);
            const float2 r = cs[e];
            const T x = from_f<T>(u * r.x - v * r.y), y = from_f<T>(v * r.x + u * r.y);
            dst[e] = x;
            dst[e + half_dims] = y;
            if (dst2) {
                dst2[e] = x;
                dst2[e + half_dims] = y;
            }
        } else {
            const int k = e + half_dims;                    // rot_dims .. rot - 1
            const T x = src[k];
            if (h < 0) dst[k] = x;
            if (dst2) dst2[k] = x;
        }
    }
}

// ---------------------------------------------------------------------------
// Absorbed form, plain FP32 kernel: one CTA per (row, head)
// ---------------------------------------------------------------------------
constexpr int kPlainThreads = 128;

template <typename T>
__global__ void __launch_bounds__(kPlainThreads)
latent_absorbed_plain_kernel(const LatentArgs<T> a, const T* __restrict__ q_abs, T* __restrict__ o_lat)
{
    extern __shared__ __align__(16) float smem[];
    constexpr int V = Vec16<T>::n;
    const int dk = a.rank + a.rot;
    float* qs = smem;                       // [dk]
    float* acc = qs + dk;                   // [rank]
    float* ps = acc + a.rank;               // [kPlainThreads]
    __shared__ float sh[kPlainThreads / 32];
    pdl_launch_dependents();
    const int row = blockIdx.x, h = blockIdx.y, b = row / a.g.seq_len, t = row - b * a.g.seq_len;
    const int tid = threadIdx.x;
    pdl_wait();
    const int limit = min((a.g.pos_dev ? *a.g.pos_dev : a.g.start_pos) + t + 1, a.max_seq);
    const T* cache = a.cache + (size_t)(a.g.first_slot + b) * a.slot_stride;
    const T* q = q_abs + ((size_t)row * a.heads + h) * dk;
    for (int i = tid; i < dk; i += kPlainThreads) qs[i] = to_f<T>(q[i]) * a.scale;
    for (int i = tid; i < a.rank; i += kPlainThreads) acc[i] = 0.f;
    float m_run = -FLT_MAX, l_run = 0.f;
    for (int k0 = 0; k0 < limit; k0 += kPlainThreads) {
        __syncthreads();
        const int k = k0 + tid;
        float s = -FLT_MAX;
        if (k < limit) {
            const uint4* kr = reinterpret_cast<const uint4*>(cache + (size_t)k * dk);
            s = 0.f;
            for (int c = 0; c < dk / V; c++) {
                float f[V];
                Vec16<T>::unpack(kr[c], f);
#pragma unroll
                for (int j = 0; j < V; j++) s = fmaf(f[j], qs[c * V + j], s);
            }
        }
        float m = warp_max(s);
        if ((tid & 31) == 0) sh[tid >> 5] = m;
        __syncthreads();
        m = fmaxf(fmaxf(sh[0], sh[1]), fmaxf(sh[2], sh[3]));
        const float m_new = fmaxf(m_run, m), corr = expf(m_run - m_new);
        const float p = k < limit ? expf(s - m_new) : 0.f;
        ps[tid] = p;
        __syncthreads();
        const float sum = warp_sum(p);
        if ((tid & 31) == 0) sh[tid >> 5] = sum;
        const int nk = min(kPlainThreads, limit - k0);
        for (int i = tid; i < a.rank; i += kPlainThreads) {
            float o = acc[i] * corr;
            for (int j = 0; j < nk; j++) o = fmaf(ps[j], to_f<T>(cache[(size_t)(k0 + j) * dk + i]), o);
            acc[i] = o;
        }
        __syncthreads();
        l_run = l_run * corr + ((sh[0] + sh[1]) + (sh[2] + sh[3]));
        m_run = m_new;
    }
    float num = 1.f;
    if (a.sink) {
        const float m = fmaxf(m_run, a.sink[h]);
        num = expf(m_run - m);
        l_run = l_run * num + expf(a.sink[h] - m);
    }
    for (int i = tid; i < a.rank; i += kPlainThreads)
        o_lat[((size_t)row * a.heads + h) * a.rank + i] = from_f<T>(acc[i] * num / l_run);
}

// ---------------------------------------------------------------------------
// Absorbed form on mma.sync: 16 (token, head) rows x one range of cache positions per CTA
// ---------------------------------------------------------------------------
constexpr int kAbsThreads = 256, kAbsWarps = kAbsThreads / 32, kAbsRows = 16;
constexpr int kAbsMaxSplit = 64, kAbsTargetCtas = 2 * 148;

struct SplitPlan {
    int row_tiles, nsplit;
};
SplitPlan split_plan(int n_seq, int seq_len, int heads, int keys)
{
    SplitPlan p;
    p.row_tiles = (seq_len * heads + kAbsRows - 1) / kAbsRows;
    int s = kAbsTargetCtas / (p.row_tiles * n_seq);
    const int most = (keys + 63) / 64;
    if (s > most) s = most;
    if (s > kAbsMaxSplit) s = kAbsMaxSplit;
    p.nsplit = s < 1 ? 1 : s;
    return p;
}

// positions per split when `total` positions exist
__device__ __forceinline__ int split_len(int total, int nsplit) { return ((total + nsplit - 1) / nsplit + 63) & ~63; }

// ws record of (sequence, row, split): rank unnormalised sums, then maximum (base-2) and sum
template <int TK, int NTW>
__global__ void __launch_bounds__(kAbsThreads)
latent_absorbed_mma_kernel(const LatentArgs<bf16> a, const bf16* __restrict__ q_abs, float* __restrict__ ws, int nsplit)
{
    extern __shared__ __align__(16) uint8_t smem_raw[];
    const int dk = a.rank + a.rot, ldk = ((dk + 15) & ~15) + 8, ksteps = (dk + 15) / 16;
    bf16* qs = reinterpret_cast<bf16*>(smem_raw);                 // [16][ldk]
    bf16* ks = qs + kAbsRows * ldk;                               // [2][TK][ldk]
    bf16* ph = ks + 2 * TK * ldk;                                 // [16][TK + 8]
    bf16* pl = ph + kAbsRows * (TK + 8);
    float* ss = reinterpret_cast<float*>(pl + kAbsRows * (TK + 8));   // [16][TK + 4]
    float* m_run = ss + kAbsRows * (TK + 4);
    float* l_run = m_run + kAbsRows;
    float* corr = l_run + kAbsRows;
    pdl_launch_dependents();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, tq = lane & 3;
    const int split = blockIdx.y, b = blockIdx.z, r0 = blockIdx.x * kAbsRows;
    const int rows = a.g.seq_len * a.heads;
    // padding columns of the tiles stay zero
    for (int i = tid; i < (kAbsRows + 2 * TK) * 16; i += kAbsThreads) {
        const int c = dk + (i & 15);
        if (c < ldk) qs[(size_t)(i >> 4) * ldk + c] = __float2bfloat16_rn(0.f);
    }
    if (tid < kAbsRows) {
        m_run[tid] = -INFINITY;
        l_run[tid] = 0.f;
    }
    pdl_wait();
    const int pos0 = a.g.pos_dev ? *a.g.pos_dev : a.g.start_pos;
    const int total = min(pos0 + a.g.seq_len, a.max_seq);
    const int len = split_len(total, nsplit), lo = split * len;
    if (lo >= total) return;
    const int last_row = min(r0 + kAbsRows, rows) - 1;
    const int hi = min(min(total, lo + len), pos0 + last_row / a.heads + 1);   // positions some row of the tile sees
    const bf16* cache = a.cache + (size_t)(a.g.first_slot + b) * a.slot_stride;
    const int pieces = dk / 8;
    const bf16* q = q_abs + ((size_t)b * rows + r0) * dk;
    for (int i = tid; i < kAbsRows * pieces; i += kAbsThreads) {
        const int r = i / pieces, c = i - r * pieces;
        const bool v = r0 + r < rows;
        cp16(qs + r * ldk + c * 8, v ? q + (size_t)r * dk + c * 8 : q_abs, v);
    }
    auto load_tile = [&](int k0, int stage) {
        bf16* dst = ks + (size_t)stage * TK * ldk;
        for (int i = tid; i < TK * pieces; i += kAbsThreads) {
            const int r = i / pieces, c = i - r * pieces;
            const bool v = k0 + r < hi;
            cp16(dst + r * ldk + c * 8, v ? cache + (size_t)(k0 + r) * dk + c * 8 : cache, v);
        }
        cp_commit();
    };
    float acc[NTW][4];
#pragma unroll
    for (int i = 0; i < NTW; i++)
#pragma unroll
        for (int e = 0; e < 4; e++) acc[i][e] = 0.f;
    const float scale2 = a.scale * kLog2e;
    const int nt = a.rank / 8;                                    // output column tiles
    if (lo < hi) load_tile(lo, 0);
    int stage = 0;
    for (int k0 = lo; k0 < hi; k0 += TK, stage ^= 1) {
        if (k0 + TK < hi) {
            load_tile(k0 + TK, stage ^ 1);
            cp_wait<1>();
        } else {
            cp_wait<0>();
        }
        __syncthreads();
        const bf16* kt = ks + (size_t)stage * TK * ldk;
        if (warp < TK / 8) {
            float c[4] = {0.f, 0.f, 0.f, 0.f};
            const bf16* qa = qs + (lane & 15) * ldk + (lane >> 4) * 8;
            const bf16* kb = kt + (warp * 8 + (lane & 7)) * ldk + ((lane >> 3) & 1) * 8;
#pragma unroll 4
            for (int k = 0; k < ksteps; k++) {
                uint32_t fa[4], fb[2];
                ldsm4(fa, qa + k * 16);
                ldsm2(fb, kb + k * 16);
                mma16816(c, fa, fb[0], fb[1]);
            }
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int r = gq + (e >> 1) * 8, n = warp * 8 + 2 * tq + (e & 1), k = k0 + n;
                const bool see = k < hi && r0 + r < rows && k <= pos0 + (r0 + r) / a.heads;
                ss[r * (TK + 4) + n] = see ? c[e] * scale2 : -INFINITY;
            }
        }
        __syncthreads();
#pragma unroll
        for (int q2 = 0; q2 < kAbsRows / kAbsWarps; q2++) {
            const int r = warp * (kAbsRows / kAbsWarps) + q2;
            float s[TK / 32], mx = -INFINITY;
#pragma unroll
            for (int j = 0; j < TK / 32; j++) {
                s[j] = ss[r * (TK + 4) + lane + 32 * j];
                mx = fmaxf(mx, s[j]);
            }
            mx = warp_max(mx);
            const float m_old = m_run[r], m_new = fmaxf(m_old, mx);
            float sum = 0.f;
#pragma unroll
            for (int j = 0; j < TK / 32; j++) {
                const float p = (s[j] == -INFINITY) ? 0.f : exp2_neg(s[j] - m_new);
                sum += p;
                const bf16 h = __float2bfloat16_rn(p);
                ph[r * (TK + 8) + lane + 32 * j] = h;
                pl[r * (TK + 8) + lane + 32 * j] = __float2bfloat16_rn(p - __bfloat162float(h));
            }
            sum = warp_sum(sum);
            __syncwarp();
            if (lane == 0) {
                const float cr = (m_old == -INFINITY) ? 0.f : exp2f(m_old - m_new);
                corr[r] = cr;
                l_run[r] = l_run[r] * cr + sum;
                m_run[r] = m_new;
            }
        }
        __syncthreads();
        const float c0 = corr[gq], c1 = corr[gq + 8];
#pragma unroll
        for (int i = 0; i < NTW; i++) {
            acc[i][0] *= c0;
            acc[i][1] *= c0;
            acc[i][2] *= c1;
            acc[i][3] *= c1;
        }
#pragma unroll
        for (int k = 0; k < TK / 16; k++) {
            uint32_t fh[4], fl[4];
            ldsm4(fh, ph + (lane & 15) * (TK + 8) + k * 16 + (lane >> 4) * 8);
            ldsm4(fl, pl + (lane & 15) * (TK + 8) + k * 16 + (lane >> 4) * 8);
#pragma unroll
            for (int i = 0; i < NTW; i++) {
                const int j = warp + kAbsWarps * i;
                if (j < nt) {
                    uint32_t fb[2];
                    ldsm2t(fb, kt + (k * 16 + (lane & 15)) * ldk + j * 8);
                    mma16816(acc[i], fh, fb[0], fb[1]);
                    mma16816(acc[i], fl, fb[0], fb[1]);
                }
            }
        }
        __syncthreads();         // the tile, the weights and the factors are rewritten next
    }
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();
    const int rec = a.rank + 2;
    float* base = ws + (((size_t)b * rows + r0) * nsplit + split) * rec;
#pragma unroll
    for (int i = 0; i < NTW; i++) {
        const int j = warp + kAbsWarps * i;
        if (j >= nt) continue;
#pragma unroll
        for (int e = 0; e < 2; e++) {
            const int r = gq + e * 8;
            if (r0 + r < rows)
                *reinterpret_cast<float2*>(base + (size_t)r * nsplit * rec + j * 8 + 2 * tq) = make_float2(acc[i][2 * e], acc[i][2 * e + 1]);
        }
    }
    if (tid < kAbsRows && r0 + tid < rows) {
        float* r = base + (size_t)tid * nsplit * rec + a.rank;
        r[0] = m_run[tid];
        r[1] = l_run[tid];
    }
}

constexpr int kMergeThreads = 64;

__global__ void __launch_bounds__(kMergeThreads)
latent_merge_kernel(const LatentArgs<bf16> a, const float* __restrict__ ws, bf16* __restrict__ o_lat, int nsplit)
{
    __shared__ float wgt[kAbsMaxSplit];
    pdl_launch_dependents();
    const int row = blockIdx.x, h = row % a.heads;      // (sequence, token, head) in order
    const int c = blockIdx.y * kMergeThreads + threadIdx.x;
    pdl_wait();
    const int total = min((a.g.pos_dev ? *a.g.pos_dev : a.g.start_pos) + a.g.seq_len, a.max_seq);
    const int len = split_len(total, nsplit), active = (total + len - 1) / len, rec = a.rank + 2;
    const float* base = ws + (size_t)row * nsplit * rec;
    // the first half of the partial sums is requested before the weights are known
    constexpr int kAtOnce = kAbsMaxSplit / 2;
    float v[kAtOnce];
    auto load = [&](int s0) {
#pragma unroll
        for (int u = 0; u < kAtOnce; u++) v[u] = (c < a.rank && s0 + u < active) ? __ldcg(base + (size_t)(s0 + u) * rec + c) : 0.f;
    };
    load(0);
    if (threadIdx.x < 32) {
        const int s0 = threadIdx.x, s1 = threadIdx.x + 32;
        const float m0 = s0 < active ? base[(size_t)s0 * rec + a.rank] : -INFINITY, m1 = s1 < active ? base[(size_t)s1 * rec + a.rank] : -INFINITY;
        float m = warp_max(fmaxf(m0, m1));
        const float sink = a.sink ? a.sink[h] * kLog2e : -INFINITY;
        m = fmaxf(m, sink);
        const float w0 = m0 == -INFINITY ? 0.f : exp2f(m0 - m), w1 = m1 == -INFINITY ? 0.f : exp2f(m1 - m);
        float l = 0.f;
        if (s0 < active) l += w0 * base[(size_t)s0 * rec + a.rank + 1];
        if (s1 < active) l += w1 * base[(size_t)s1 * rec + a.rank + 1];
        l = warp_sum(l);
        if (a.sink) l += exp2f(sink - m);
        wgt[s0] = w0 / l;
        wgt[s1] = w1 / l;
    }
    __syncthreads();
    if (c >= a.rank) return;
    float o = 0.f;
    for (int s0 = 0; s0 < active; s0 += kAtOnce) {
        if (s0) load(s0);
#pragma unroll
        for (int u = 0; u < kAtOnce; u++)
            if (s0 + u < active) o = fmaf(wgt[s0 + u], v[u], o);
    }
    o_lat[(size_t)row * a.rank + c] = __float2bfloat16_rn(o);
}

size_t absorbed_smem(int tk, int dk)
{
    const size_t ldk = ((size_t)(dk + 15) / 16) * 16 + 8;
    return ((kAbsRows + 2 * tk) * ldk + 2 * kAbsRows * (tk + 8)) * sizeof(bf16) + (kAbsRows * (tk + 4) + 3 * kAbsRows) * sizeof(float);
}

// ---------------------------------------------------------------------------
// Expanded form on mma.sync: 64 queries of one head per CTA, tiles of 64 positions
// ---------------------------------------------------------------------------
constexpr int kExpWarps = 4, kExpThreads = kExpWarps * 32, kExpQ = 16 * kExpWarps, kExpK = 64;

template <int NV>      // 8-wide output column tiles, even
__global__ void __launch_bounds__(kExpThreads)
latent_expanded_kernel(const LatentArgs<bf16> a, const bf16* __restrict__ kx, const bf16* __restrict__ vx, bf16* __restrict__ out)
{
    extern __shared__ __align__(16) uint8_t smem_raw[];
    const int dq = a.dim + a.rot, ldq = ((dq + 15) & ~15) + 8, ksteps = (dq + 15) / 16;
    const int ldv = ((a.vdim + 15) & ~15) + 8, nv = (a.vdim + 15) / 16 * 2;
    bf16* qs = reinterpret_cast<bf16*>(smem_raw);               // [64][ldq]
    bf16* ks = qs + kExpQ * ldq;                                // [2][64][ldq]
    bf16* vs = ks + 2 * kExpK * ldq;                            // [2][64][ldv]
    pdl_launch_dependents();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, tq = lane & 3;
    const int h = blockIdx.y, q0 = (gridDim.x - 1 - blockIdx.x) * kExpQ;       // longest first
    for (int i = tid; i < (kExpQ + 2 * kExpK) * 16; i += kExpThreads) {
        const int c = dq + (i & 15);
        if (c < ldq) qs[(size_t)(i >> 4) * ldq + c] = __float2bfloat16_rn(0.f);
    }
    for (int i = tid; i < 2 * kExpK * 16; i += kExpThreads) {
        const int c = a.vdim + (i & 15);
        if (c < ldv) vs[(size_t)(i >> 4) * ldv + c] = __float2bfloat16_rn(0.f);
    }
    pdl_wait();
    const int pos0 = a.g.start_pos, n = a.g.seq_len;
    const int nq = min(kExpQ, n - q0), hi = pos0 + q0 + nq;     // positions [0, hi) are seen by some query of the tile
    const int dk = a.rank + a.rot;
    const bf16* cache = a.cache + (size_t)a.g.first_slot * a.slot_stride;
    {
        const int pieces = dq / 8;
        for (int i = tid; i < kExpQ * pieces; i += kExpThreads) {
            const int r = i / pieces, c = i - r * pieces;
            const bool v = r < nq;
            cp16(qs + r * ldq + c * 8, v ? a.proj + (size_t)(q0 + r) * a.ld + a.q_off + (size_t)h * dq + c * 8 : a.proj, v);
        }
    }
    // pieces of 16 bytes per row: unrotated key, shared key part, value; i / pieces as a multiplication
    const int pk = a.dim / 8, pr = a.rot / 8, pv = a.vdim / 8;
    const uint32_t mk = 0xffffffffu / pk + 1, mr = pr ? 0xffffffffu / pr + 1 : 0, mv = 0xffffffffu / pv + 1;
    const bf16 *kxh = kx + (size_t)h * a.dim, *vxh = vx + (size_t)h * a.vdim, *krh = cache + a.rank;
    const size_t kx_ld = (size_t)a.heads * a.dim, vx_ld = (size_t)a.heads * a.vdim;
    auto load_part = [&](bf16* dst, int ld, const bf16* src, size_t src_ld, int pieces, uint32_t magic, int k0) {
        for (int i = tid; i < kExpK * pieces; i += kExpThreads) {
            const int r = pieces == 1 ? i : (int)__umulhi((uint32_t)i, magic), c = (i - r * pieces) * 8;
            const bool v = k0 + r < hi;
            cp16(dst + r * ld + c, v ? src + (size_t)(k0 + r) * src_ld + c : src, v);
        }
    };
    auto load_tile = [&](int k0, int stage) {
        bf16 *kd = ks + (size_t)stage * kExpK * ldq, *vd = vs + (size_t)stage * kExpK * ldv;
        load_part(kd, ldq, kxh, kx_ld, pk, mk, k0);
        if (pr) load_part(kd + a.dim, ldq, krh, (size_t)dk, pr, mr, k0);
        load_part(vd, ldv, vxh, vx_ld, pv, mv, k0);
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
    load_tile(0, 0);
    int stage = 0;
    for (int k0 = 0; k0 < hi; k0 += kExpK, stage ^= 1) {
        if (k0 + kExpK < hi) {
            load_tile(k0 + kExpK, stage ^ 1);
            cp_wait<1>();
        } else {
            cp_wait<0>();
        }
        __syncthreads();
        const bf16 *kt = ks + (size_t)stage * kExpK * ldq, *vt = vs + (size_t)stage * kExpK * ldv;
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
        const bool edge = k0 + kExpK > pos0 + q0 + 1;          // some (query, position) pair of the tile is masked
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int j = 0; j < 8; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                float v = s[j][e] * scale2;
                if (edge && k0 + j * 8 + 2 * tq + (e & 1) > pos0 + q0 + row + (e >> 1) * 8) v = -INFINITY;
                s[j][e] = v;
                mx[e >> 1] = fmaxf(mx[e >> 1], v);
            }
        float cr[2];
#pragma unroll
        for (int e = 0; e < 2; e++) {
            mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 1));
            mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 2));
            const float m_new = fmaxf(m_run[e], mx[e]);
            cr[e] = exp2_neg(m_run[e] - m_new);                // 0 at first: position 0 is seen by every query
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
                    v[e] = exp2_neg(v[e] - m_run[e >> 1]);
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
        float num = 1.f;
        if (a.sink) {
            const float sink = a.sink[h] * kLog2e, m = fmaxf(m_run[e], sink);
            num = exp2f(m_run[e] - m);
            l = l * num + exp2f(sink - m);
        }
        const int r = row + e * 8;
        if (r >= nq) continue;
        float f = num / l;
        if (a.gate) f *= sigmoid_f(__bfloat162float(a.gate[(size_t)(q0 + r) * a.gate_ld + h]));
        bf16* op = out + ((size_t)(q0 + r) * a.heads + h) * a.vdim;
#pragma unroll
        for (int j = 0; j < NV; j++) {
            const int c = j * 8 + 2 * tq;
            if (c < a.vdim)
                *reinterpret_cast<__nv_bfloat162*>(op + c) = __floats2bfloat162_rn(o[j][2 * e] * f, o[j][2 * e + 1] * f);
        }
    }
}

size_t expanded_smem(int dq, int vdim)
{
    const size_t ldq = ((size_t)(dq + 15) / 16) * 16 + 8, ldv = ((size_t)(vdim + 15) / 16) * 16 + 8;
    return ((kExpQ + 2 * kExpK) * ldq + 2 * kExpK * ldv) * sizeof(bf16);
}

constexpr size_t kSmemLimit = 220 * 1024;

template <typename K>
int allow_smem(K kernel)
{
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSmemLimit) != cudaSuccess)
        return fail(TLLM_ERR_LAUNCH, "latent attention: %s", cudaGetErrorString(cudaGetLastError()));
    return TLLM_OK;
}

template <typename T>
int check_latent(const LatentArgs<T>& a)
{
    if (a.heads < 1 || a.dim % 8 || a.rot % 8 || a.vdim % 8 || a.rank % 8 || a.rank < 8 || a.rot_dims % 2 || a.rot_dims > a.rot || a.ld % 8 ||
        a.q_off % 8 || a.kv_off % 8)
        return fail(TLLM_ERR_SHAPE, "latent attention: heads=%d dim=%d rot=%d(%d) vdim=%d rank=%d", a.heads, a.dim, a.rot, a.rot_dims, a.vdim, a.rank);
    if (!a.g.pos_dev && a.g.start_pos + a.g.seq_len > a.max_seq)
        return fail(TLLM_ERR_SHAPE, "latent attention: positions %d..%d beyond the cache (%d)", a.g.start_pos, a.g.start_pos + a.g.seq_len - 1, a.max_seq);
    return TLLM_OK;
}

template <int TK>
int launch_absorbed_tk(const LatentArgs<bf16>& a, const bf16* q_abs, float* ws, SplitPlan p, cudaStream_t stream)
{
    const dim3 grid(p.row_tiles, p.nsplit, a.g.n_seq), block(kAbsThreads);
    const size_t smem = absorbed_smem(TK, a.rank + a.rot);
    const int per_warp = (a.rank / 8 + kAbsWarps - 1) / kAbsWarps;
    int st;
#define TLLM_CASE(N)                                                                                                        \
    if (per_warp <= N) {                                                                                                     \
        if ((st = allow_smem(latent_absorbed_mma_kernel<TK, N>))) return st;                                                 \
        return launch_pdl("latent_absorbed", latent_absorbed_mma_kernel<TK, N>, grid, block, smem, stream, a, q_abs, ws, p.nsplit); \
    }
    TLLM_CASE(1)
    TLLM_CASE(2)
    TLLM_CASE(4)
    TLLM_CASE(8)
    TLLM_CASE(16)
#undef TLLM_CASE
    return fail(TLLM_ERR_SHAPE, "latent attention: rank=%d", a.rank);
}

template <typename T>
int launch_plain(const LatentArgs<T>& a, const T* q_abs, T* o_lat, cudaStream_t stream)
{
    const size_t smem = (size_t)(2 * a.rank + a.rot + kPlainThreads) * sizeof(float);
    if (smem > kSmemLimit) return fail(TLLM_ERR_SHAPE, "latent attention: rank=%d rot=%d", a.rank, a.rot);
    int st = allow_smem(latent_absorbed_plain_kernel<T>);
    if (st) return st;
    return launch_pdl("latent_absorbed_plain", latent_absorbed_plain_kernel<T>, dim3(a.g.rows(), a.heads), dim3(kPlainThreads), smem, stream,
                      a, q_abs, o_lat);
}

int absorbed(const LatentArgs<float>& a, const float* q_abs, float* o_lat, float*, cudaStream_t stream)
{
    return launch_plain<float>(a, q_abs, o_lat, stream);
}

int absorbed(const LatentArgs<bf16>& a, const bf16* q_abs, bf16* o_lat, float* ws, cudaStream_t stream)
{
    const int dk = a.rank + a.rot;
    const bool fits64 = absorbed_smem(64, dk) <= kSmemLimit, fits32 = absorbed_smem(32, dk) <= kSmemLimit;
    if (!fits32 || a.rank > 8 * kAbsWarps * 16) return launch_plain<bf16>(a, q_abs, o_lat, stream);
    const SplitPlan p = split_plan(a.g.n_seq, a.g.seq_len, a.heads, a.g.pos_dev ? a.max_seq : a.g.start_pos + a.g.seq_len);
    int st = fits64 ? launch_absorbed_tk<64>(a, q_abs, ws, p, stream) : launch_absorbed_tk<32>(a, q_abs, ws, p, stream);
    if (st) return st;
    return launch_pdl("latent_merge", latent_merge_kernel, dim3(a.g.rows() * a.heads, (a.rank + kMergeThreads - 1) / kMergeThreads),
                      dim3(kMergeThreads), 0, stream, a, ws, o_lat, p.nsplit);
}

}  // namespace

template <typename T>
int launch_latent_prep(const LatentArgs<T>& a, T* q_abs, cudaStream_t stream)
{
    if (a.g.rows() == 0) return TLLM_OK;
    int st = check_latent(a);
    if (st) return st;
    return launch_pdl("latent_prep", latent_prep_kernel<T>, dim3(a.g.rows(), 2), dim3(kPrepThreads), 0, stream, a, q_abs);
}
template int launch_latent_prep<bf16>(const LatentArgs<bf16>&, bf16*, cudaStream_t);
template int launch_latent_prep<float>(const LatentArgs<float>&, float*, cudaStream_t);

size_t latent_workspace_floats(int rows, int heads, int rank)
{
    // rows * heads * nsplit records; split_plan keeps row tiles * nsplit at kAbsTargetCtas or at one split
    const size_t tiles = ((size_t)rows * heads + kAbsRows - 1) / kAbsRows + rows;
    const size_t recs = (tiles > kAbsTargetCtas ? tiles : (size_t)kAbsTargetCtas) * kAbsRows;
    return recs * (rank + 2);
}

template <typename T>
int launch_latent_absorbed(const LatentArgs<T>& a, const T* q_abs, T* o_lat, float* ws, cudaStream_t stream)
{
    if (a.g.rows() == 0) return TLLM_OK;
    int st = check_latent(a);
    if (st) return st;
    return absorbed(a, q_abs, o_lat, ws, stream);
}
template int launch_latent_absorbed<bf16>(const LatentArgs<bf16>&, const bf16*, bf16*, float*, cudaStream_t);
template int launch_latent_absorbed<float>(const LatentArgs<float>&, const float*, float*, float*, cudaStream_t);

bool latent_expanded_supported(const LatentArgs<bf16>& a)
{
    return a.g.n_seq == 1 && !a.g.pos_dev && a.vdim <= 256 && expanded_smem(a.dim + a.rot, a.vdim) <= kSmemLimit;
}

int launch_latent_expanded(const LatentArgs<bf16>& a, const bf16* kx, const bf16* vx, bf16* out, cudaStream_t stream)
{
    if (a.g.rows() == 0) return TLLM_OK;
    int st = check_latent(a);
    if (st) return st;
    if (!latent_expanded_supported(a)) return fail(TLLM_ERR_SHAPE, "latent attention: no expanded form for dim=%d rot=%d vdim=%d", a.dim, a.rot, a.vdim);
    const dim3 grid((a.g.seq_len + kExpQ - 1) / kExpQ, a.heads), block(kExpThreads);
    const size_t smem = expanded_smem(a.dim + a.rot, a.vdim);
#define TLLM_CASE(N)                                                                                                     \
    if (a.vdim <= 8 * N) {                                                                                                \
        if ((st = allow_smem(latent_expanded_kernel<N>))) return st;                                                      \
        return launch_pdl("latent_expanded", latent_expanded_kernel<N>, grid, block, smem, stream, a, kx, vx, out);        \
    }
    TLLM_CASE(4)
    TLLM_CASE(8)
    TLLM_CASE(16)
    TLLM_CASE(32)
#undef TLLM_CASE
    return TLLM_ERR_SHAPE;
}

}  // namespace tllm
