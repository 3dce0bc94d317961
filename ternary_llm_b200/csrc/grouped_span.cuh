// Device code of grouped-query attention that several kernels share: norms and rotation of a head,
// one query row against a range of positions, the merge of such ranges.
#pragma once
#include <cfloat>

#include "launch.cuh"
#include "mixers.cuh"
#include "mma_sync.cuh"

namespace tllm {

namespace {

constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ int first_seen(int pos, int chunk) { return chunk > 0 ? pos / chunk * chunk : 0; }

// One head's vector by one warp: norm, rotation; put(entry, value)
template <typename T, typename F>
__device__ __forceinline__ void norm_rotate(const T* x, const GroupedArgs<T>& a, const float* w, int pos, F&& put)
{
    const int lane = threadIdx.x & 31, half = a.rot_dims >> 1;
    const float2* cs = a.rope + (size_t)pos * half;
    float f = 1.f;
    if (w) {
        float ss = 0.f;
        for (int i = lane; i < a.dim; i += 32) {
            const float v = to_f<T>(x[i]);
            ss += v * v;
        }
        f = 1.0f / sqrtf(warp_sum(ss) / (float)a.dim_true + a.eps);
    }
    auto at = [&](int i) { return to_f<T>(x[i]) * (w ? f * w[i] : 1.f); };
    for (int i = lane; i < half; i += 32) {
        const float u = at(i), v = at(i + half);
        const float2 r = cs[i];
        put(i, u * r.x - v * r.y);
        put(i + half, v * r.x + u * r.y);
    }
    for (int i = a.rot_dims + lane; i < a.dim; i += 32) put(i, at(i));
}

// The same with eight neighbouring entries per lane, `lanes` lanes per vector (a power of two, lane
// l of them): put(first entry, values).  Needs rot_dims in steps of 16 and dim <= 8 * lanes.
__device__ __forceinline__ void load8(const bf16* p, float (&v)[8]) { Vec16<bf16>::unpack(*reinterpret_cast<const uint4*>(p), v); }
__device__ __forceinline__ void load8(const float* p, float (&v)[8])
{
    Vec16<float>::unpack(*reinterpret_cast<const uint4*>(p), v);
    Vec16<float>::unpack(*reinterpret_cast<const uint4*>(p + 4), v + 4);
}
__device__ __forceinline__ void store8(bf16* p, const float (&v)[8])
{
    __nv_bfloat162 t[4];
#pragma unroll
    for (int i = 0; i < 4; i++) t[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    *reinterpret_cast<uint4*>(p) = *reinterpret_cast<const uint4*>(t);
}
__device__ __forceinline__ void store8(float* p, const float (&v)[8])
{
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
template <typename T> __host__ __device__ __forceinline__ bool rotates8(const GroupedArgs<T>& a) { return a.rot_dims % 16 == 0 && a.dim <= 256; }

template <typename T, typename F>
__device__ __forceinline__ void norm_rotate8(const T* x, const GroupedArgs<T>& a, const float* w, int pos, int lanes, int l, F&& put)
{
    const int half = a.rot_dims >> 1, half8 = half >> 3;
    const bool in = l * 8 < a.dim, turns = l < 2 * half8;
    float v[8], g[8], c[16];
#pragma unroll
    for (int j = 0; j < 8; j++) v[j] = g[j] = 0.f;
    if (in) load8(x + l * 8, v);
    if (in && w) load8(w + l * 8, g);
    if (turns) {
        const float* cs = reinterpret_cast<const float*>(a.rope + (size_t)pos * half + (l < half8 ? l : l - half8) * 8);
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const float4 t = *reinterpret_cast<const float4*>(cs + 4 * j);
            c[4 * j] = t.x;
            c[4 * j + 1] = t.y;
            c[4 * j + 2] = t.z;
            c[4 * j + 3] = t.w;
        }
    }
    if (w) {
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < 8; j++) ss += v[j] * v[j];
        for (int o = lanes >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        const float f = 1.0f / sqrtf(ss / (float)a.dim_true + a.eps);
#pragma unroll
        for (int j = 0; j < 8; j++) v[j] = v[j] * (f * g[j]);
    }
    const int partner = (int)(threadIdx.x & 31) + (!turns ? 0 : l < half8 ? half8 : -half8);
#pragma unroll
    for (int j = 0; j < 8; j++) {
        const float o = __shfl_sync(0xffffffffu, v[j], partner);
        if (turns) v[j] = l < half8 ? v[j] * c[2 * j] - o * c[2 * j + 1] : v[j] * c[2 * j] + o * c[2 * j + 1];
    }
    if (in) put(l * 8, v);
}

// ---------------------------------------------------------------------------
// One query row against a range of positions
// ---------------------------------------------------------------------------
constexpr int kSpanThreads = 256, kSpanWarps = kSpanThreads / 32, kSpanHeads = 8;
constexpr int kSpanAcc = 4;                          // pairs of output entries per thread
constexpr int kSpanMaxSplit = 32, kSpanTargetCtas = 2 * 148;

__device__ __forceinline__ int range_len(int span, int nsplit, int tile) { return ((span + tile - 1) / tile + nsplit - 1) / nsplit * tile; }

template <typename T> __device__ __forceinline__ float2 pair_of(const T* p);
template <> __device__ __forceinline__ float2 pair_of<bf16>(const bf16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }
template <> __device__ __forceinline__ float2 pair_of<float>(const float* p) { return *reinterpret_cast<const float2*>(p); }

__device__ __forceinline__ void copy16(void* dst, const void* src, bool valid)
{
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(sm32(dst)), "l"(src), "r"(valid ? 16 : 0) : "memory");
}

// One CTA: row, (key/value head, head block), split.  ws record of (row, head, split): vdim unnormalised
// sums, maximum, sum.  ONE: a single new token per sequence, not yet in the cache.
template <typename T, int TK, bool ONE>
__device__ __forceinline__ void grouped_span(const GroupedArgs<T>& a, float* __restrict__ ws, int hb, int blocks, uint8_t* smem_raw, int row, int by,
                                             int split, int nsplit)
{
    constexpr int V = Vec16<T>::n, PAD = V, SETS = kSpanThreads / TK, MAXH = (kSpanHeads + SETS - 1) / SETS;
    const int D = a.dim, E = a.vdim, ldk = D + PAD;
    float* qs = reinterpret_cast<float*>(smem_raw);                  // [hb][D], times the scale
    float* ps = qs + hb * D;                                          // [hb][TK]
    T* kt = reinterpret_cast<T*>(ps + hb * TK);                       // [TK][ldk]
    T* vt = kt + TK * ldk;                                            // [TK][E]
    __shared__ float m_s[kSpanHeads], l_s[kSpanHeads], c_s[kSpanHeads];
    const int b = row / a.g.seq_len, t = row - b * a.g.seq_len;
    const int g = by / blocks, per = a.heads / a.kv_heads, h0 = (by - g * blocks) * hb;
    const int nh = min(hb, per - h0);                                 // query heads g * per + h0 ..
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int pos = (a.g.pos_dev ? *a.g.pos_dev : a.g.start_pos) + t;
    if (pos >= a.max_seq) return;
    const int first = first_seen(pos, a.chunk), len = range_len(pos + 1 - first, nsplit, TK);
    const int p0 = first + split * len, p1 = min(pos + 1, p0 + len);
    if (p0 >= p1) return;
    const T* proj = a.proj + (size_t)row * a.ld;
    T* kc = a.kc + (size_t)(a.g.first_slot + b) * a.k_slot + (size_t)g * D;
    T* vc = a.vc + (size_t)(a.g.first_slot + b) * a.v_slot + (size_t)g * E;
    const size_t krow = (size_t)a.kv_heads * D, vrow = (size_t)a.kv_heads * E;
    const int stored = ONE ? pos : pos + 1;                           // positions before it are in the cache
    auto load = [&](int k0) {
        // a row per warp and turn, its key pieces and then its value pieces
        const int nk = D / V, nv = E / V, base = k0 % a.cache_rows;
        for (int r = warp; r < TK; r += kSpanWarps) {
            const int p = k0 + r;
            if (ONE && p == pos) continue;                            // written below
            const bool v = p < p1 && p < stored;
            int ring = base + r;
            if (v && ring >= a.cache_rows) ring -= a.cache_rows;
            const T *ksrc = v ? kc + (size_t)ring * krow : kc, *vsrc = v ? vc + (size_t)ring * vrow : vc;
            T *kdst = kt + r * ldk, *vdst = vt + r * E;
            for (int c = lane; c < nk + nv; c += 32) {
                if (c < nk) copy16(kdst + c * V, v ? ksrc + c * V : kc, v);
                else copy16(vdst + (c - nk) * V, v ? vsrc + (c - nk) * V : vc, v);
            }
        }
        cp_commit();
        if (ONE && pos >= k0 && pos < k0 + TK && pos < p1) {          // the new token's key and value, here and into the cache
            const int r = pos - k0, ring = pos % a.cache_rows;
            T *krow_s = kt + r * ldk, *krow_g = kc + (size_t)ring * krow;
            if (warp == kSpanWarps - 1) {
                const T* src = proj + a.k_off + (size_t)g * D;
                if (rotates8(a))
                    norm_rotate8<T>(src, a, a.k_norm, pos, 32, lane, [&](int i, const float (&v)[8]) {
                        store8(krow_s + i, v);
                        if (h0 == 0) store8(krow_g + i, v);
                    });
                else
                    norm_rotate<T>(src, a, a.k_norm, pos, [&](int i, float v) {
                        krow_s[i] = from_f<T>(v);
                        if (h0 == 0) krow_g[i] = from_f<T>(v);
                    });
            } else {
                for (int i = tid; i < E; i += kSpanThreads - 32) {
                    const T v = proj[a.v_off + (size_t)g * E + i];
                    vt[r * E + i] = v;
                    if (h0 == 0) vc[(size_t)ring * vrow + i] = v;
                }
            }
        }
    };
    load(p0);
    for (int h = warp; h < nh; h += kSpanWarps) {
        const T* q = proj + a.q_off + (size_t)(g * per + h0 + h) * D;
        if (ONE && rotates8(a))
            norm_rotate8<T>(q, a, a.q_norm, pos, 32, lane, [&](int i, const float (&v)[8]) {
#pragma unroll
                for (int j = 0; j < 8; j++) qs[h * D + i + j] = to_f<T>(from_f<T>(v[j])) * a.scale;
            });
        else if (ONE) norm_rotate<T>(q, a, a.q_norm, pos, [&](int i, float v) { qs[h * D + i] = to_f<T>(from_f<T>(v)) * a.scale; });
        else
            for (int i = lane; i < D; i += 32) qs[h * D + i] = to_f<T>(q[i]) * a.scale;
    }
    if (tid < kSpanHeads) {
        m_s[tid] = -FLT_MAX;
        l_s[tid] = 0.f;
    }
    float2 acc[kSpanAcc];
#pragma unroll
    for (int j = 0; j < kSpanAcc; j++) acc[j] = make_float2(0.f, 0.f);
    const int e2 = E >> 1, outs = nh * e2;
    for (int k0 = p0; k0 < p1; k0 += TK) {
        cp_wait<0>();
        __syncthreads();
        {
            const int r = tid & (TK - 1), set = tid / TK;             // one position, every SETS-th head
            float s[MAXH];
#pragma unroll
            for (int j = 0; j < MAXH; j++) s[j] = 0.f;
#pragma unroll 2
            for (int c = 0; c < D; c += V) {
                float kf[V];
                Vec16<T>::unpack(*reinterpret_cast<const uint4*>(kt + r * ldk + c), kf);
#pragma unroll
                for (int j = 0; j < MAXH; j++) {
                    const int h = set + j * SETS;
                    if (h >= nh) break;
                    const float4* q = reinterpret_cast<const float4*>(qs + h * D + c);
#pragma unroll
                    for (int u = 0; u < V / 4; u++) {
                        const float4 x = q[u];
                        s[j] = fmaf(kf[4 * u], x.x, fmaf(kf[4 * u + 1], x.y, fmaf(kf[4 * u + 2], x.z, fmaf(kf[4 * u + 3], x.w, s[j]))));
                    }
                }
            }
#pragma unroll
            for (int j = 0; j < MAXH; j++)
                if (set + j * SETS < nh) ps[(set + j * SETS) * TK + r] = k0 + r < p1 ? s[j] : -FLT_MAX;
        }
        __syncthreads();
        for (int h = warp; h < nh; h += kSpanWarps) {
            float mx = -FLT_MAX;
            for (int i = lane; i < TK; i += 32) mx = fmaxf(mx, ps[h * TK + i]);
            const float m = fmaxf(m_s[h], warp_max(mx));
            float sum = 0.f;
            for (int i = lane; i < TK; i += 32) {
                const float p = k0 + i < p1 ? expf(ps[h * TK + i] - m) : 0.f;
                ps[h * TK + i] = p;
                sum += p;
            }
            sum = warp_sum(sum);
            __syncwarp();
            if (lane == 0) {
                const float c = expf(m_s[h] - m);
                c_s[h] = c;
                l_s[h] = l_s[h] * c + sum;
                m_s[h] = m;
            }
        }
        __syncthreads();
        const int nk = min(TK, p1 - k0);
#pragma unroll
        for (int j = 0; j < kSpanAcc; j++) {
            const int o = tid + j * kSpanThreads;
            if (o >= outs) break;
            const int h = o / e2, c = (o - h * e2) * 2;
            const float f = c_s[h];
            float2 s = make_float2(acc[j].x * f, acc[j].y * f);
#pragma unroll 8
            for (int i = 0; i < nk; i++) {
                const float p = ps[h * TK + i];
                const float2 v = pair_of<T>(vt + i * E + c);
                s.x = fmaf(p, v.x, s.x);
                s.y = fmaf(p, v.y, s.y);
            }
            acc[j] = s;
        }
        __syncthreads();
        if (k0 + TK < p1) load(k0 + TK);
    }
#pragma unroll
    for (int j = 0; j < kSpanAcc; j++) {
        const int o = tid + j * kSpanThreads;
        if (o >= outs) break;
        const int h = o / e2, c = (o - h * e2) * 2, head = g * per + h0 + h;
        if (nsplit == 1) {
            const float f = a.out_scale / l_s[h];
            T* op = a.out + (size_t)row * a.ld_out + (size_t)head * E + c;
            op[0] = from_f<T>(acc[j].x * f);
            op[1] = from_f<T>(acc[j].y * f);
        } else {
            float* rec = ws + (((size_t)row * a.heads + head) * nsplit + split) * (E + 2);
            rec[c] = acc[j].x;
            rec[c + 1] = acc[j].y;
            if (c == 0) {
                rec[E] = m_s[h];
                rec[E + 1] = l_s[h];
            }
        }
    }
}

// Partial results of one (row, head); wgt: kSpanMaxSplit words
template <typename T, int TK>
__device__ __forceinline__ void grouped_merge(const GroupedArgs<T>& a, const float* __restrict__ ws, int nsplit, int row, int h, float* wgt)
{
    constexpr int kAtOnce = 16;
    const int t = row % a.g.seq_len, c0 = threadIdx.x;
    const size_t ld = a.vdim + 2;
    const float* rec = ws + ((size_t)row * a.heads + h) * nsplit * ld;
    // the records are requested before it is known how many of them count
    float v[kAtOnce], m = -FLT_MAX, l = 0.f;
#pragma unroll
    for (int s = 0; s < kAtOnce; s++) v[s] = (s < nsplit && c0 < a.vdim) ? rec[s * ld + c0] : 0.f;
    if (threadIdx.x < nsplit) {
        m = rec[threadIdx.x * ld + a.vdim];
        l = rec[threadIdx.x * ld + a.vdim + 1];
    }
    const int pos = (a.g.pos_dev ? *a.g.pos_dev : a.g.start_pos) + t;
    if (pos >= a.max_seq) return;
    const int span = pos + 1 - first_seen(pos, a.chunk), len = range_len(span, nsplit, TK), n = (span + len - 1) / len;
    if (threadIdx.x < 32) {
        const bool counts = threadIdx.x < n;
        const float mx = warp_max(counts ? m : -FLT_MAX), e = counts ? expf(m - mx) : 0.f, sum = warp_sum(counts ? e * l : 0.f);
        wgt[threadIdx.x] = e * a.out_scale / sum;
    }
    __syncthreads();
    for (int c = c0; c < a.vdim; c += blockDim.x) {
        float o = 0.f;
#pragma unroll
        for (int s = 0; s < kAtOnce; s++)
            if (s < n) o = fmaf(wgt[s], c == c0 ? v[s] : rec[s * ld + c], o);
        for (int s = kAtOnce; s < n; s++) o = fmaf(wgt[s], rec[s * ld + c], o);
        a.out[(size_t)row * a.ld_out + (size_t)h * a.vdim + c] = from_f<T>(o);
    }
}

constexpr size_t kSmemLimit = 220 * 1024;

struct SpanPlan {
    int hb, blocks, nsplit, tk;
    size_t smem;
};
size_t span_smem(int hb, int dim, int vdim, int tk, size_t es)
{
    return (size_t)hb * (dim + tk) * 4 + (size_t)tk * (dim + 16 / es + vdim) * es;
}
SpanPlan span_plan(int rows, int heads, int kv_heads, int dim, int vdim, int max_seq, int chunk, size_t es)
{
    SpanPlan p;
    const int per = heads / kv_heads, fit = kSpanAcc * 2 * kSpanThreads / vdim;
    p.hb = per < fit ? per : fit;
    if (p.hb > kSpanHeads) p.hb = kSpanHeads;
    if (p.hb < 1) p.hb = 1;
    p.blocks = (per + p.hb - 1) / p.hb;
    p.tk = span_smem(p.hb, dim, vdim, 64, es) <= kSmemLimit / 2 ? 64 : 16;
    p.smem = span_smem(p.hb, dim, vdim, p.tk, es);
    const int span = chunk > 0 && chunk < max_seq ? chunk : max_seq;
    int s = kSpanTargetCtas / (rows * kv_heads * p.blocks);
    const int most = (span + p.tk - 1) / p.tk;
    if (s > most) s = most;
    if (s > kSpanMaxSplit) s = kSpanMaxSplit;
    p.nsplit = s < 1 ? 1 : s;
    return p;
}

template <typename T>
int check_grouped(const GroupedArgs<T>& a)
{
    if (!grouped_supported(a.heads, a.kv_heads, a.dim, a.vdim) || a.rot_dims < 0 || a.rot_dims % 2 || a.rot_dims > a.dim || a.ld % 8 || a.q_off % 8 ||
        a.k_off % 8 || a.v_off % 8 || a.ld_out % 2 || a.cache_rows < 1)
        return fail(TLLM_ERR_SHAPE, "grouped attention: heads=%d/%d dim=%d vdim=%d rot=%d", a.heads, a.kv_heads, a.dim, a.vdim, a.rot_dims);
    if (!a.g.pos_dev && a.g.start_pos + a.g.seq_len > a.max_seq)
        return fail(TLLM_ERR_SHAPE, "grouped attention: positions %d..%d beyond the cache (%d)", a.g.start_pos, a.g.start_pos + a.g.seq_len - 1, a.max_seq);
    return TLLM_OK;
}

}  // namespace

}  // namespace tllm
