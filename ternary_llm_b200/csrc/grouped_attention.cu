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

// grid (rows, kv_heads * head blocks, splits).  ws record of (row, head, split): vdim unnormalised
// sums, maximum, sum.  ONE: a single new token per sequence, not yet in the cache.
template <typename T, int TK, bool ONE>
__global__ void __launch_bounds__(kSpanThreads)
grouped_span_kernel(const GroupedArgs<T> a, float* __restrict__ ws, int hb, int blocks)
{
    extern __shared__ __align__(16) uint8_t smem_raw[];
    constexpr int V = Vec16<T>::n, PAD = V, SETS = kSpanThreads / TK, MAXH = (kSpanHeads + SETS - 1) / SETS;
    const int D = a.dim, E = a.vdim, ldk = D + PAD, nsplit = gridDim.z, split = blockIdx.z;
    float* qs = reinterpret_cast<float*>(smem_raw);                  // [hb][D], times the scale
    float* ps = qs + hb * D;                                          // [hb][TK]
    T* kt = reinterpret_cast<T*>(ps + hb * TK);                       // [TK][ldk]
    T* vt = kt + TK * ldk;                                            // [TK][E]
    __shared__ float m_s[kSpanHeads], l_s[kSpanHeads], c_s[kSpanHeads];
    pdl_launch_dependents();
    const int row = blockIdx.x, b = row / a.g.seq_len, t = row - b * a.g.seq_len;
    const int g = blockIdx.y / blocks, per = a.heads / a.kv_heads, h0 = (blockIdx.y - g * blocks) * hb;
    const int nh = min(hb, per - h0);                                 // query heads g * per + h0 ..
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    pdl_wait();
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
        const int nk = D / V, nv = E / V;
        for (int i = tid; i < TK * nk; i += kSpanThreads) {
            const int r = i / nk, c = i - r * nk, p = k0 + r;
            const bool v = p < p1 && p < stored;
            if (ONE && p == pos) continue;                            // written below
            copy16(kt + r * ldk + c * V, v ? kc + (size_t)(p % a.cache_rows) * krow + c * V : kc, v);
        }
        for (int i = tid; i < TK * nv; i += kSpanThreads) {
            const int r = i / nv, c = i - r * nv, p = k0 + r;
            const bool v = p < p1 && p < stored;
            if (ONE && p == pos) continue;
            copy16(vt + r * E + c * V, v ? vc + (size_t)(p % a.cache_rows) * vrow + c * V : vc, v);
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

constexpr int kMergeThreads = 128;

template <typename T, int TK>
__global__ void __launch_bounds__(kMergeThreads)
grouped_merge_kernel(const GroupedArgs<T> a, const float* __restrict__ ws, int nsplit)
{
    __shared__ float wgt[kSpanMaxSplit];
    pdl_launch_dependents();
    const int row = blockIdx.x, h = blockIdx.y, t = row % a.g.seq_len;
    pdl_wait();
    const int pos = (a.g.pos_dev ? *a.g.pos_dev : a.g.start_pos) + t;
    if (pos >= a.max_seq) return;
    const int span = pos + 1 - first_seen(pos, a.chunk), len = range_len(span, nsplit, TK), n = (span + len - 1) / len;
    const float* rec = ws + ((size_t)row * a.heads + h) * nsplit * (a.vdim + 2);
    if (threadIdx.x < 32) {
        const int s = threadIdx.x;
        const float m = s < n ? rec[(size_t)s * (a.vdim + 2) + a.vdim] : -FLT_MAX, mx = warp_max(m);
        const float e = s < n ? expf(m - mx) : 0.f, l = warp_sum(s < n ? e * rec[(size_t)s * (a.vdim + 2) + a.vdim + 1] : 0.f);
        wgt[s] = e * a.out_scale / l;
    }
    __syncthreads();
    for (int c = threadIdx.x; c < a.vdim; c += kMergeThreads) {
        float o = 0.f;
#pragma unroll 8
        for (int s = 0; s < n; s++) o = fmaf(wgt[s], rec[(size_t)s * (a.vdim + 2) + c], o);
        a.out[(size_t)row * a.ld_out + (size_t)h * a.vdim + c] = from_f<T>(o);
    }
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

constexpr size_t kSmemLimit = 220 * 1024;
constexpr int kPromptFrom = 16;       // tokens from which the tensor-core kernel runs

size_t prompt_smem(int dim, int vdim)
{
    const size_t ldq = ((size_t)(dim + 15) / 16) * 16 + 8, ldv = ((size_t)(vdim + 15) / 16) * 16 + 8;
    return ((kPq + 2 * kPk) * ldq + 2 * kPk * ldv) * sizeof(bf16);
}

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
    if (!grouped_supported(a.heads, a.kv_heads, a.dim, a.vdim) || a.rot_dims < 0 || a.rot_dims % 2 || a.rot_dims > a.dim || a.ld % 8 || a.q_off % 8 ||
        a.k_off % 8 || a.v_off % 8 || a.ld_out % 2 || a.cache_rows < 1)
        return fail(TLLM_ERR_SHAPE, "grouped attention: heads=%d/%d dim=%d vdim=%d rot=%d", a.heads, a.kv_heads, a.dim, a.vdim, a.rot_dims);
    if (!a.g.pos_dev && a.g.start_pos + a.g.seq_len > a.max_seq)
        return fail(TLLM_ERR_SHAPE, "grouped attention: positions %d..%d beyond the cache (%d)", a.g.start_pos, a.g.start_pos + a.g.seq_len - 1, a.max_seq);
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
