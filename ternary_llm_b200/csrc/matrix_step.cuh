// Device code of the matrix recurrences that several kernels share: the token-by-token form and the
// gated norm of an output row.
#pragma once
#include <cooperative_groups.h>

#include "launch.cuh"
#include "mixers.cuh"

namespace tllm {

namespace {

constexpr float kUnitEps = 1e-6f;     // under the root of the unit vectors

__device__ __forceinline__ float log_decay(float a, float dt_bias, float neg_a) { return neg_a * softplus_f(a + dt_bias); }

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

// ---------------------------------------------------------------------------
// Token by token
// ---------------------------------------------------------------------------
constexpr int kSeqThreads = 256, kSeqMaxCluster = 8, kSeqStates = 16, kSeqTokens = 8;   // entries of a column per lane; tokens staged together

// A column of S is spread over `lpc` lanes in pieces of four entries; a CTA serves blockDim / lpc
// columns of one head.
// (bx, h, b): column block, head, sequence.
template <typename T, bool DELTA>
__device__ __forceinline__ void matrix_seq(const MatrixScanArgs<T>& a, int lpc, float* smem, int bx, int h, int b)
{
    constexpr int NP = kSeqStates / 4;
    const int cols = blockDim.x / lpc, D = a.dim, D4 = D >> 2;
    float* ks = smem;                                   // [tokens][D]
    float* qs = ks + kSeqTokens * D;
    float* vs = qs + kSeqTokens * D;                    // [tokens][cols]
    float* gs = vs + kSeqTokens * cols;                 // decay, step size
    float* bs = gs + kSeqTokens;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, warps = blockDim.x >> 5;
    const int cl = tid / lpc, l = tid - cl * lpc, c0 = bx * cols, c = c0 + cl;
    const int kh = h / (a.heads / a.kv_heads);
    const bool live = c < a.vdim;
    float4* st = reinterpret_cast<float4*>(a.state + (size_t)(a.g.first_slot + b) * a.slot_stride + ((size_t)h * a.vdim + (live ? c : 0)) * D);
    float4 S[NP];
#pragma unroll
    for (int u = 0; u < NP; u++) {
        const int p = l + u * lpc;
        S[u] = p < D4 ? st[p] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const bool fresh = (a.g.pos_dev ? *a.g.pos_dev : a.g.start_pos) == 0;
    if (fresh || !live) {
#pragma unroll
        for (int u = 0; u < NP; u++) S[u] = make_float4(0.f, 0.f, 0.f, 0.f);
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

// A single new token per sequence, the same layout of a column over lanes: everything a thread needs
// is requested at once, and the lanes of a column find the vectors' lengths among themselves.
// NORM (the CTAs of a head form a cluster): the head's output goes through its norm and gate here;
// sh: 16 words of shared memory.
template <typename T, bool DELTA, bool NORM>
__device__ __forceinline__ void matrix_one(const MatrixScanArgs<T>& a, const GatedNormArgs<T>& norm, int log_lpc, float* sh, int bx, int h, int b)
{
    constexpr int NP = kSeqStates / 4;
    const int tid = threadIdx.x, lane = tid & 31, D = a.dim, D4 = D >> 2, lpc = 1 << log_lpc;
    if (NORM && gridDim.x > 1) cooperative_groups::this_cluster().barrier_arrive();
    const int l = tid & (lpc - 1), c = bx * (blockDim.x >> log_lpc) + (tid >> log_lpc);
    const bool live = c < a.vdim;
    const int col = live ? c : 0, kh = a.kv_heads == a.heads ? h : h / (a.heads / a.kv_heads);
    float4* st = reinterpret_cast<float4*>(a.state + (size_t)(a.g.first_slot + b) * a.slot_stride + ((size_t)h * a.vdim + col) * D);
    const T *kp = a.k + (size_t)b * a.ld + (size_t)kh * D, *qp = a.q + (size_t)b * a.ld + (size_t)kh * D;
    float4 S[NP], k[NP], q[NP];
#pragma unroll
    for (int u = 0; u < NP; u++) {
        const int p = l + (u << log_lpc);
        const bool in = p < D4;
        S[u] = in ? st[p] : make_float4(0.f, 0.f, 0.f, 0.f);
        k[u] = in ? get4(kp + 4 * p) : make_float4(0.f, 0.f, 0.f, 0.f);
        q[u] = in ? get4(qp + 4 * p) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    float add = to_f<T>(a.v[(size_t)b * a.ld + (size_t)h * a.vdim + col]);
    const size_t ab = (size_t)b * a.ld_ab + h;
    float g, beta = 0.f, gate = 0.f, weight = 0.f;
    if (DELTA) {
        beta = a.b[ab];
        g = log_decay(a.a[ab], a.dt_bias[h], a.neg_a[h]);
    } else {
        g = a.decay[h];
    }
    if (NORM) {
        gate = to_f<T>(norm.gate[(size_t)b * norm.ld_gate + (size_t)h * a.vdim + col]);
        weight = norm.w[col];
    }
    const bool fresh = (a.g.pos_dev ? *a.g.pos_dev : a.g.start_pos) == 0;
    if (fresh) {
#pragma unroll
        for (int u = 0; u < NP; u++) S[u] = make_float4(0.f, 0.f, 0.f, 0.f);
    }
    float fq = 1.f;
    if (DELTA) {
        beta = sigmoid_f(beta);
        g = decay_exp(g, expf(g));
        float kk = 0.f, qq = 0.f, p = 0.f;
#pragma unroll
        for (int u = 0; u < NP; u++) {
            kk += (k[u].x * k[u].x + k[u].y * k[u].y) + (k[u].z * k[u].z + k[u].w * k[u].w);
            qq += (q[u].x * q[u].x + q[u].y * q[u].y) + (q[u].z * q[u].z + q[u].w * q[u].w);
        }
        for (int o = lpc >> 1; o > 0; o >>= 1) {
            kk += __shfl_xor_sync(0xffffffffu, kk, o);
            qq += __shfl_xor_sync(0xffffffffu, qq, o);
        }
        const float fk = 1.f / sqrtf(kk + kUnitEps);
        fq = a.q_scale / sqrtf(qq + kUnitEps);
#pragma unroll
        for (int u = 0; u < NP; u++) {
            k[u].x *= fk;
            k[u].y *= fk;
            k[u].z *= fk;
            k[u].w *= fk;
            S[u].x *= g;
            S[u].y *= g;
            S[u].z *= g;
            S[u].w *= g;
            p = fmaf(S[u].x, k[u].x, fmaf(S[u].y, k[u].y, fmaf(S[u].z, k[u].z, fmaf(S[u].w, k[u].w, p))));
        }
        for (int o = lpc >> 1; o > 0; o >>= 1) p += __shfl_xor_sync(0xffffffffu, p, o);
        add = beta * (add - p);
    }
    float o = 0.f;
#pragma unroll
    for (int u = 0; u < NP; u++) {
        const float d = DELTA ? 1.f : g;
        S[u].x = fmaf(k[u].x, add, d * S[u].x);
        S[u].y = fmaf(k[u].y, add, d * S[u].y);
        S[u].z = fmaf(k[u].z, add, d * S[u].z);
        S[u].w = fmaf(k[u].w, add, d * S[u].w);
        o = fmaf(S[u].x, q[u].x, fmaf(S[u].y, q[u].y, fmaf(S[u].z, q[u].z, fmaf(S[u].w, q[u].w, o))));
        if (live && l + (u << log_lpc) < D4) st[l + (u << log_lpc)] = S[u];
    }
    for (int s = lpc >> 1; s > 0; s >>= 1) o += __shfl_xor_sync(0xffffffffu, o, s);
    o *= fq;
    if (!NORM) {
        if (live && l == 0) a.o[((size_t)b * a.heads + h) * a.vdim + c] = o;
        return;
    }
    float ss = warp_sum(l == 0 && live ? o * o : 0.f);           // each column counts once
    const int warps = blockDim.x >> 5;
    if (lane == 0) sh[tid >> 5] = ss;
    __syncthreads();
    ss = 0.f;
    for (int i = 0; i < warps; i++) ss += sh[i];
    if (gridDim.x > 1) {
        cooperative_groups::cluster_group cluster = cooperative_groups::this_cluster();
        cluster.barrier_wait();                                  // the others are running, their shared memory is there
        if (tid < (int)gridDim.x) cluster.map_shared_rank(sh, tid)[8 + bx] = ss;
        cluster.sync();
        ss = 0.f;
        for (int i = 0; i < (int)gridDim.x; i++) ss += sh[8 + i];
    }
    if (live && l == 0)
        norm.out[(size_t)b * norm.ld_out + (size_t)h * a.vdim + c] =
            from_f<T>(o * (norm.out_scale / sqrtf(ss / (float)norm.n_true + norm.eps)) * weight * apply_act(norm.act, gate));
}

struct SeqPlan {
    int lpc, log_lpc, threads, blocks;
    size_t smem;
};
inline size_t seq_smem(int dim, int cols) { return (size_t)kSeqTokens * (2 * dim + cols + 2) * sizeof(float); }
inline SeqPlan seq_plan(int dim, int vdim)
{
    SeqPlan p;
    p.lpc = 1;
    p.log_lpc = 0;
    while (p.lpc * kSeqStates < dim) {
        p.lpc *= 2;
        p.log_lpc++;
    }
    p.threads = kSeqThreads;
    const int cols = p.threads / p.lpc;
    p.blocks = (vdim + cols - 1) / cols;
    p.smem = seq_smem(dim, cols);
    return p;
}

template <typename T>
int check_matrix_scan(const MatrixScanArgs<T>& a)
{
    if (a.heads < 1 || a.kv_heads < 1 || a.heads % a.kv_heads || a.dim < 8 || a.dim % 8 || a.dim > 512 || a.vdim < 8 || a.vdim % 8 || a.ld % 8 ||
        (a.delta ? !a.a || !a.b || !a.neg_a || !a.dt_bias : !a.decay))
        return fail(TLLM_ERR_SHAPE, "matrix_scan: heads=%d/%d dim=%d (8..512) vdim=%d ld=%d", a.heads, a.kv_heads, a.dim, a.vdim, a.ld);
    return TLLM_OK;
}

// ---------------------------------------------------------------------------
// Gated norm
// ---------------------------------------------------------------------------
constexpr int kGnThreads = 256, kGnWarps = kGnThreads / 32;

// One row by a CTA; sh: kGnWarps words; a warp per group, or the whole CTA when the row is one group
template <typename T>
__device__ __forceinline__ void gated_norm_row(const GatedNormArgs<T>& a, int row, float* sh)
{
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const bool whole = a.groups == 1;
    const int step = whole ? kGnThreads : 32, i0 = whole ? tid : lane, n4 = a.n >> 2;
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

}  // namespace tllm
