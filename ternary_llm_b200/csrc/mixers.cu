// Residual chain, causal convolution and the two recurrences of the mixed-layer decoder.
//
// A recurrence over many tokens is cut into time chunks: a first launch runs every chunk but the
// last from a zero state and records its final state and its total decay, a second one derives
// each chunk's true initial state from the records before it and produces the outputs.  The
// first launch also copies the carried state into the records: in the second one the last chunk
// overwrites it while others may not have started.  Short portions and single tokens are one
// chunk and need the second launch only.
#include "launch.cuh"
#include "mixers.cuh"

namespace tllm {

namespace {

__device__ __forceinline__ float cta_sum(float v, float* sh)
{
    v = warp_sum(v);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) sh[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.f;
    for (int i = 0; i < (int)(blockDim.x >> 5); i++) t += sh[i];     // same order in every thread
    return t;
}

__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const bf16* p)
{
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16),
                       __uint_as_float(v.y & 0xffff0000u));
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(bf16* p, float4 v)
{
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}
__device__ __forceinline__ float sq4(float4 v) { return (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w); }

constexpr int kNormThreads = 256;

template <typename T>
__global__ void __launch_bounds__(kNormThreads)
norm_chain_kernel(const NormArgs<T> a)
{
    extern __shared__ __align__(16) float vals[];      // [w]
    __shared__ float sh[kNormThreads / 32];
    pdl_launch_dependents();
    pdl_wait();
    const int row = blockIdx.x, src = a.row_map ? a.row_map[row] : row;
    const int n4 = a.w >> 2;
    float* x = a.x + (size_t)src * a.w;
    float rinv = 1.f;
    auto branch = [&](int i) -> float4 {                // this row's y
        if (!a.parts) return load4(a.y + (size_t)row * a.w + 4 * i);
        float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
        for (int k = 0; k < a.top; k++) {
            const float4 v = load4(a.parts + (size_t)a.part_row[(size_t)row * a.top + k] * a.w + 4 * i);
            const float p = a.part_w[(size_t)row * a.top + k];
            s.x = fmaf(p, v.x, s.x);
            s.y = fmaf(p, v.y, s.y);
            s.z = fmaf(p, v.z, s.z);
            s.w = fmaf(p, v.w, s.w);
        }
        return s;
    };
    const bool any = a.y || a.parts;
    if (any && a.w_post) {
        float ss = 0.f;
        for (int i = threadIdx.x; i < n4; i += kNormThreads) {
            const float4 v = branch(i);
            store4(vals + 4 * i, v);
            ss += sq4(v);
        }
        rinv = 1.0f / sqrtf(cta_sum(ss, sh) / (float)a.width + a.eps);
    }
    float ss = 0.f;
    auto finish = [&](int i, float4 v) {                // the new residual
        if (a.tap) {
            const float t[4] = {v.x, v.y, v.z, v.w};
            for (int j = 0; j < 4; j++)
                if (4 * i + j < a.tap_width) a.tap[(size_t)row * a.tap_width + 4 * i + j] = t[j];
        }
        if (a.extra) {
            const float4 e = load4(a.extra + (size_t)row * a.w + 4 * i);
            v.x += e.x;
            v.y += e.y;
            v.z += e.z;
            v.w += e.w;
        }
        if (!a.row_map) store4(x + 4 * i, v);
        store4(vals + 4 * i, v);
        ss += sq4(v);
    };
    for (int i = threadIdx.x; i < n4; i += kNormThreads) {
        float4 v;
        if (a.table) {
            v = load4(a.table + (size_t)a.tokens[row] * a.w + 4 * i);
            if (a.emb) store4(a.emb + (size_t)row * a.w + 4 * i, v);
        } else {
            v = load4(x + 4 * i);
        }
        if (any) {
            float4 y, w = make_float4(1.f, 1.f, 1.f, 1.f);
            if (a.w_post) {
                y = load4(vals + 4 * i);
                w = load4(a.w_post + 4 * i);
            } else {
                y = branch(i);
            }
            v.x = a.alpha * v.x + y.x * rinv * w.x;
            v.y = a.alpha * v.y + y.y * rinv * w.y;
            v.z = a.alpha * v.z + y.z * rinv * w.z;
            v.w = a.alpha * v.w + y.w * rinv * w.w;
        }
        if (a.w_sum) {
            store4(vals + 4 * i, v);
            ss += sq4(v);
        } else {
            finish(i, v);
        }
    }
    if (a.w_sum) {
        rinv = 1.0f / sqrtf(cta_sum(ss, sh) / (float)a.width + a.eps);
        ss = 0.f;
        for (int i = threadIdx.x; i < n4; i += kNormThreads) {
            const float4 v = load4(vals + 4 * i), w = load4(a.w_sum + 4 * i);
            finish(i, make_float4(v.x * rinv * w.x, v.y * rinv * w.y, v.z * rinv * w.z, v.w * rinv * w.w));
        }
    }
    if (!a.h) return;
    if (!a.w_next) {
        for (int i = threadIdx.x; i < n4; i += kNormThreads) store4(a.h + (size_t)row * a.w + 4 * i, load4(vals + 4 * i));
        return;
    }
    rinv = 1.0f / sqrtf(cta_sum(ss, sh) / (float)a.width + a.eps);
    for (int i = threadIdx.x; i < n4; i += kNormThreads) {
        const float4 v = load4(vals + 4 * i), w = load4(a.w_next + 4 * i);
        store4(a.h + (size_t)row * a.w + 4 * i, make_float4(v.x * rinv * w.x, v.y * rinv * w.y, v.z * rinv * w.z, v.w * rinv * w.w));
    }
}

// ---------------------------------------------------------------------------
// Causal convolution per channel
// ---------------------------------------------------------------------------
constexpr int kConvThreads = 128, kConvChunk = 32;

template <typename T> struct Pair;
template <> struct Pair<bf16> { using type = __nv_bfloat162; };
template <> struct Pair<float> { using type = float2; };
__device__ __forceinline__ float2 ld2(const bf16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }
__device__ __forceinline__ float2 ld2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ void st2(bf16* p, float2 v) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v.x, v.y); }
__device__ __forceinline__ void st2(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }

// A thread owns two adjacent channels and one time chunk; only the threads of the first chunk
// read the carried inputs, and they also write the new ones.  TAPS = 0: any number of taps.
template <typename T, int TAPS>
__global__ void __launch_bounds__(kConvThreads)
causal_conv_kernel(const ConvArgs<T> a, int chunk)
{
    pdl_launch_dependents();
    const int c = 2 * (blockIdx.x * kConvThreads + threadIdx.x), b = blockIdx.z;
    const int taps = TAPS ? TAPS : a.taps, n = a.g.seq_len;
    const int t0 = blockIdx.y * chunk, t1 = min(n, t0 + chunk);
    pdl_wait();
    if (c >= a.channels) return;
    const bool fresh = (a.g.pos_dev ? *a.g.pos_dev : a.g.start_pos) == 0;
    const T* x = a.x + (size_t)b * n * a.ldx + c;
    T* y = a.y + (size_t)b * n * a.channels + c;
    T* st = a.state + (size_t)(a.g.first_slot + b) * a.slot_stride + c;
    const float b0 = a.bias ? a.bias[c] : 0.f, b1 = a.bias ? a.bias[c + 1] : 0.f;
    auto input = [&](int s) -> float2 {                    // input of token s (s < 0: carried)
        if (s >= 0) return ld2(x + (size_t)s * a.ldx);
        return fresh ? make_float2(0.f, 0.f) : ld2(st + (size_t)(taps - 1 + s) * a.channels);
    };
    if (TAPS) {
        float w0[TAPS ? TAPS : 1], w1[TAPS ? TAPS : 1];
        float2 win[TAPS ? TAPS : 1];
#pragma unroll
        for (int j = 0; j < TAPS; j++) {
            w0[j] = a.w[(size_t)c * TAPS + j];
            w1[j] = a.w[(size_t)(c + 1) * TAPS + j];
        }
#pragma unroll
        for (int j = 1; j < TAPS; j++) win[j] = input(t0 - TAPS + j);
#pragma unroll 8
        for (int t = t0; t < t1; t++) {
#pragma unroll
            for (int j = 0; j + 1 < TAPS; j++) win[j] = win[j + 1];
            win[TAPS - 1] = ld2(x + (size_t)t * a.ldx);
            float v0 = b0, v1 = b1;
#pragma unroll
            for (int j = 0; j < TAPS; j++) {
                v0 = fmaf(w0[j], win[j].x, v0);
                v1 = fmaf(w1[j], win[j].y, v1);
            }
            st2(y + (size_t)t * a.channels, make_float2(apply_act(a.act, v0), apply_act(a.act, v1)));
        }
    } else {
        for (int t = t0; t < t1; t++) {
            float v0 = b0, v1 = b1;
            for (int j = 0; j < taps; j++) {
                const float2 v = input(t - taps + 1 + j);
                v0 = fmaf(a.w[(size_t)c * taps + j], v.x, v0);
                v1 = fmaf(a.w[(size_t)(c + 1) * taps + j], v.y, v1);
            }
            st2(y + (size_t)t * a.channels, make_float2(apply_act(a.act, v0), apply_act(a.act, v1)));
        }
    }
    // ascending: entry j is taken from token n - taps + 1 + j, i.e. from a carried entry after j
    if (t0 == 0)
        for (int j = 0; j + 1 < taps; j++) st2(st + (size_t)j * a.channels, input(n - taps + 1 + j));
}

// ---------------------------------------------------------------------------
// Selective scan
// ---------------------------------------------------------------------------
constexpr int kScanThreads = 128;
constexpr int kMaxChunks = 16, kMinChunk = 32;     // time chunks; tokens of a chunk at least

// a state of many entries per channel makes records expensive: fewer chunks
inline int time_chunks(int n, int states)
{
    const int c = n / kMinChunk, most = states > 1 ? kMaxChunks : 2 * kMaxChunks;
    return c < 1 ? 1 : c > most ? most : c;
}

// A channel is served by `lpc` lanes with NS states each; lane l holds states l * NS ...  B and C
// of TT tokens are staged in shared memory as floats, the channel's own inputs in registers.
// Records of chunk k: [b][k][state][channel] final states, then [b][k][channel] sums of dt.
// ONE: lpc is 1.  DT: the step sizes are computed here too (few tokens: one launch less).
template <typename T, int NS, int TT, bool OUT, bool ONE, bool DT>
__global__ void __launch_bounds__(kScanThreads, 4)
selective_scan_kernel(const ScanArgs<T> a, int lanes, int nchunk)
{
    const int lpc = ONE ? 1 : lanes;
    extern __shared__ __align__(16) float bcs[];               // [TT][2][sp]
    pdl_launch_dependents();
    const int sp = lpc * NS, cpb = kScanThreads / lpc;
    const int tid = threadIdx.x, cl = tid / lpc, l = tid - cl * lpc, s0 = l * NS;
    const int c_raw = blockIdx.x * cpb + cl, chunk = blockIdx.y, b = blockIdx.z;
    const bool live = c_raw < a.channels;
    const int c = live ? c_raw : a.channels - 1;
    const int n = a.g.seq_len, len = (n + nchunk - 1) / nchunk, t0 = min(n, chunk * len), t1 = min(n, t0 + len);
    float A[NS], S[NS];
#pragma unroll
    for (int j = 0; j < NS; j++) {
        A[j] = (s0 + j < a.states) ? a.a2[(size_t)c * a.states + s0 + j] : 0.f;
        S[j] = 0.f;
    }
    const float D = (OUT && a.d) ? a.d[c] : 0.f;
    const float dt_bias = (DT && a.dt_bias) ? a.dt_bias[c] : 0.f;
    pdl_wait();
    const size_t row0 = (size_t)b * n, CH = a.channels;
    const float* dtp = a.dt + row0 * CH + c;
    const T* xp = a.x + row0 * CH + c;
    const T* zp = a.z ? a.z + row0 * a.ld_z + c : nullptr;
    T* yp = a.y + row0 * CH + c;
    float* stp = a.state + (size_t)(a.g.first_slot + b) * a.slot_stride + (size_t)c * a.states;
    float* rec = a.rec + (size_t)b * nchunk * a.states * CH + c;
    float* rec_dt = a.rec + (size_t)a.g.n_seq * nchunk * a.states * CH + (size_t)b * nchunk * CH + c;
    const bool fresh = (a.g.pos_dev ? *a.g.pos_dev : a.g.start_pos) == 0;
    // the carried state as slot nchunk - 1 of the records (free: that chunk records nothing)
    float* carried = rec + (size_t)(nchunk - 1) * a.states * CH;
    if (!OUT && chunk == 0 && live) {
#pragma unroll
        for (int j = 0; j < NS; j++)
            if (s0 + j < a.states) carried[(size_t)(s0 + j) * CH] = fresh ? 0.f : stp[s0 + j];
    }
    if (OUT) {
#pragma unroll
        for (int j = 0; j < NS; j++)
            if (s0 + j < a.states) S[j] = nchunk > 1 ? carried[(size_t)(s0 + j) * CH] : fresh ? 0.f : stp[s0 + j];
#pragma unroll 2
        for (int k = 0; k < chunk; k++) {
            const float d = rec_dt[(size_t)k * CH];
#pragma unroll
            for (int j = 0; j < NS; j++)
                if (s0 + j < a.states) S[j] = fmaf(decay_exp2<T>(d * A[j]), S[j], rec[((size_t)k * a.states + s0 + j) * CH]);
        }
    }
    float sum_dt = 0.f;
    // inputs of the next TT tokens, requested one tile ahead; B and C too when a channel is one
    // lane (a handful of values per thread then)
    constexpr int NB = ONE ? TT * 2 * NS / kScanThreads : 1;
    float dt_n[TT], x_n[TT], z_n[OUT ? TT : 1], bc_n[NB];
    auto bc_at = [&](int t, int i) -> float {
        const int u = i / (2 * sp), r = i - u * 2 * sp, s = r < sp ? r : r - sp;
        return (t + u < t1 && s < a.states) ? to_f<T>(a.bc[(row0 + t + u) * a.ld_bc + (r < sp ? a.b_off : a.c_off) + s]) : 0.f;
    };
    auto request = [&](int t) {
#pragma unroll
        for (int u = 0; u < TT; u++) {                         // past the end dt = x = 0: the state stays
            const bool in = t + u < t1;
            if (!DT) dt_n[u] = in ? dtp[(size_t)(t + u) * CH] : 0.f;
            x_n[u] = in ? to_f<T>(xp[(size_t)(t + u) * CH]) : 0.f;
            if (OUT) z_n[u] = (in && zp) ? to_f<T>(zp[(size_t)(t + u) * a.ld_z]) : 0.f;
        }
        if (ONE) {
#pragma unroll
            for (int j = 0; j < NB; j++) bc_n[j] = bc_at(t, tid + j * kScanThreads);
        }
    };
    request(t0);
    for (int t = t0; t < t1; t += TT) {
        float dt[TT], x[TT], z[OUT ? TT : 1];
#pragma unroll
        for (int u = 0; u < TT; u++) {
            x[u] = x_n[u];
            if (OUT) z[u] = z_n[u];
            if (DT) {
                float p = 0.f;
                const uint4* wp = reinterpret_cast<const uint4*>(a.dt_w + (size_t)c * a.dt_rank);
                const uint4* vp = reinterpret_cast<const uint4*>(a.bc + (row0 + min(t + u, n - 1)) * a.ld_bc + a.dt_off);
                for (int i = l; i < a.dt_rank / Vec16<T>::n; i += lpc) {
                    float wf[Vec16<T>::n], vf[Vec16<T>::n];
                    Vec16<T>::unpack(__ldg(wp + i), wf);
                    Vec16<T>::unpack(vp[i], vf);
#pragma unroll
                    for (int j = 0; j < Vec16<T>::n; j++) p = fmaf(wf[j], vf[j], p);
                }
                for (int o = lpc >> 1; o > 0; o >>= 1) p += __shfl_xor_sync(0xffffffffu, p, o);
                dt[u] = t + u < t1 ? softplus_f(p + dt_bias) : 0.f;
            } else {
                dt[u] = dt_n[u];
            }
        }
        __syncthreads();
        if (ONE) {
#pragma unroll
            for (int j = 0; j < NB; j++) bcs[tid + j * kScanThreads] = bc_n[j];
        } else {
            for (int i = tid; i < TT * 2 * sp; i += kScanThreads) bcs[i] = bc_at(t, i);
        }
        __syncthreads();
        if (t + TT < t1) request(t + TT);
        float y[TT];
#pragma unroll
        for (int u = 0; u < TT; u++) {
            const float dx = dt[u] * x[u];
            const float* Bp = bcs + u * 2 * sp + s0;
            float y0 = 0.f, y1 = 0.f;
            if (!OUT) sum_dt += dt[u];
#pragma unroll
            for (int j = 0; j < NS; j += 4) {
                const float4 Bv = load4(Bp + j);
                S[j] = fmaf(decay_exp2<T>(dt[u] * A[j]), S[j], dx * Bv.x);
                S[j + 1] = fmaf(decay_exp2<T>(dt[u] * A[j + 1]), S[j + 1], dx * Bv.y);
                S[j + 2] = fmaf(decay_exp2<T>(dt[u] * A[j + 2]), S[j + 2], dx * Bv.z);
                S[j + 3] = fmaf(decay_exp2<T>(dt[u] * A[j + 3]), S[j + 3], dx * Bv.w);
                if (OUT) {
                    const float4 Cv = load4(Bp + sp + j);
                    y0 = fmaf(S[j], Cv.x, y0);
                    y1 = fmaf(S[j + 1], Cv.y, y1);
                    y0 = fmaf(S[j + 2], Cv.z, y0);
                    y1 = fmaf(S[j + 3], Cv.w, y1);
                }
            }
            y[u] = y0 + y1;
        }
        if (OUT) {
            if (!ONE)
                for (int o = lpc >> 1; o > 0; o >>= 1) {
#pragma unroll
                    for (int u = 0; u < TT; u++) y[u] += __shfl_xor_sync(0xffffffffu, y[u], o);
                }
            if (live && l == 0) {
#pragma unroll
                for (int u = 0; u < TT; u++) {
                    float v = fmaf(D, x[u], y[u]);
                    if (zp) v *= z[u] * sigmoid_f(z[u]);
                    if (t + u < t1) yp[(size_t)(t + u) * CH] = from_f<T>(v);
                }
            }
        }
    }
    if (!live) return;
    if (OUT) {
        if (chunk == nchunk - 1) {
#pragma unroll
            for (int j = 0; j < NS; j++)
                if (s0 + j < a.states) stp[s0 + j] = S[j];
        }
    } else {
#pragma unroll
        for (int j = 0; j < NS; j++)
            if (s0 + j < a.states) rec[((size_t)chunk * a.states + s0 + j) * CH] = S[j];
        if (l == 0) rec_dt[(size_t)chunk * CH] = sum_dt;
    }
}

// ---------------------------------------------------------------------------
// Real-gated linear recurrence: one thread per channel and time chunk
// ---------------------------------------------------------------------------
constexpr int kGateThreads = 64;

template <typename T, bool OUT>
__global__ void __launch_bounds__(kGateThreads)
gated_scan_kernel(const GatedScanArgs<T> a, int nchunk)
{
    constexpr int TT = 8;
    pdl_launch_dependents();
    const int c = blockIdx.x * kGateThreads + threadIdx.x, chunk = blockIdx.y, b = blockIdx.z;
    const int n = a.g.seq_len, len = (n + nchunk - 1) / nchunk, t0 = min(n, chunk * len), t1 = min(n, t0 + len);
    const float kc = c < a.channels ? -a.c * a.soft_lam[c] : 0.f;
    pdl_wait();
    if (c >= a.channels) return;
    const size_t row0 = (size_t)b * n, CH = a.channels;
    const int blk = c / a.block, ci = c - blk * a.block;
    const float* rp = a.gates + row0 * 2 * CH + (size_t)blk * 2 * a.block + ci;
    const T* up = a.u + row0 * CH + c;
    const T* yp = a.y + row0 * a.ld_y + c;
    T* op = a.out + row0 * CH + c;
    float* stp = a.state + (size_t)(a.g.first_slot + b) * a.slot_stride + c;
    float* rec = a.rec + (size_t)b * nchunk * CH + c;
    float* rec_log = a.rec + (size_t)(a.g.n_seq + b) * nchunk * CH + c;
    float S = 0.f, sum_log = 0.f;
    const bool fresh = (a.g.pos_dev ? *a.g.pos_dev : a.g.start_pos) == 0;
    float* carried = rec + (size_t)(nchunk - 1) * CH;          // see selective_scan_kernel
    if (!OUT && chunk == 0) *carried = fresh ? 0.f : *stp;
    if (OUT) {
        S = nchunk > 1 ? *carried : fresh ? 0.f : *stp;
#pragma unroll 8
        for (int k = 0; k < chunk; k++) S = fmaf(expf(rec_log[(size_t)k * CH]), S, rec[(size_t)k * CH]);
    }
    for (int t = t0; t < t1; t += TT) {
        float r[TT], i[TT], u[TT], y[OUT ? TT : 1];
#pragma unroll
        for (int j = 0; j < TT; j++) {
            const bool in = t + j < t1;                        // past the end r = u = 0: the state stays
            r[j] = in ? rp[(size_t)(t + j) * 2 * CH] : 0.f;
            i[j] = in ? rp[(size_t)(t + j) * 2 * CH + a.block] : 0.f;
            u[j] = in ? to_f<T>(up[(size_t)(t + j) * CH]) : 0.f;
            if (OUT) y[j] = in ? to_f<T>(yp[(size_t)(t + j) * a.ld_y]) : 0.f;
        }
        if (OUT) apply_act_n(a.act, y);
#pragma unroll
        for (int j = 0; j < TT; j++) {
            const float log_a = kc * r[j], A = decay_exp(log_a, expf(log_a));
            if (!OUT) sum_log += log_a;
            S = fmaf(A, S, sqrtf(one_minus_exp(2.f * log_a, A * A)) * i[j] * u[j]);
            if (OUT && t + j < t1) op[(size_t)(t + j) * CH] = from_f<T>(S * y[j]);
        }
    }
    if (OUT) {
        if (chunk == nchunk - 1) *stp = S;
    } else {
        rec[(size_t)chunk * CH] = S;
        rec_log[(size_t)chunk * CH] = sum_log;
    }
}

}  // namespace

template <typename T>
int launch_norm_chain(const NormArgs<T>& a, cudaStream_t stream)
{
    if (a.rows == 0) return TLLM_OK;
    const size_t smem = (size_t)a.w * sizeof(float);
    if (a.w % 8 || a.w < a.width || smem > 200 * 1024) return fail(TLLM_ERR_SHAPE, "norm_chain: width=%d padded to %d", a.width, a.w);
    static bool attr[64] = {};
    int dev = 0;
    cudaGetDevice(&dev);
    if (!attr[dev]) {
        cudaFuncSetAttribute(norm_chain_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        attr[dev] = true;
    }
    return launch_pdl("norm_chain", norm_chain_kernel<T>, dim3(a.rows), dim3(kNormThreads), smem, stream, a);
}

template <typename T>
int launch_causal_conv(const ConvArgs<T>& a, cudaStream_t stream)
{
    if (a.g.rows() == 0) return TLLM_OK;
    if (a.channels % 2 || a.ldx % 2 || a.taps < 1) return fail(TLLM_ERR_SHAPE, "causal_conv: channels=%d ldx=%d taps=%d", a.channels, a.ldx, a.taps);
    const int chunk = a.taps - 1 > kConvChunk ? a.taps - 1 : kConvChunk;
    const dim3 grid((a.channels / 2 + kConvThreads - 1) / kConvThreads, (a.g.seq_len + chunk - 1) / chunk, a.g.n_seq), block(kConvThreads);
    switch (a.taps) {
        case 2: return launch_pdl("causal_conv", causal_conv_kernel<T, 2>, grid, block, 0, stream, a, chunk);
        case 3: return launch_pdl("causal_conv", causal_conv_kernel<T, 3>, grid, block, 0, stream, a, chunk);
        case 4: return launch_pdl("causal_conv", causal_conv_kernel<T, 4>, grid, block, 0, stream, a, chunk);
        default: return launch_pdl("causal_conv", causal_conv_kernel<T, 0>, grid, block, 0, stream, a, chunk);
    }
}

size_t scan_record_floats(int n_seq, int seq_len, int channels, int states)
{
    const int nchunk = time_chunks(seq_len, states);
    return nchunk > 1 ? (size_t)n_seq * nchunk * channels * (states + 1) : 0;
}

namespace {
template <typename T, int NS, int TT, bool ONE, bool DT>
int scan_passes(const ScanArgs<T>& a, int lpc, int nchunk, cudaStream_t stream)
{
    const int cpb = kScanThreads / lpc;
    const size_t smem = (size_t)TT * 2 * lpc * NS * sizeof(float);
    const auto first = selective_scan_kernel<T, NS, TT, false, ONE, DT>, second = selective_scan_kernel<T, NS, TT, true, ONE, DT>;
    if (smem > 48 * 1024) {
        cudaFuncSetAttribute(first, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        cudaFuncSetAttribute(second, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    }
    const unsigned gx = (a.channels + cpb - 1) / cpb;
    if (nchunk > 1) {
        // the last chunk's final state is nobody's initial state
        const int st = launch_pdl("selective_scan", first, dim3(gx, nchunk - 1, a.g.n_seq), dim3(kScanThreads), smem, stream, a, lpc, nchunk);
        if (st) return st;
    }
    return launch_pdl("selective_scan", second, dim3(gx, nchunk, a.g.n_seq), dim3(kScanThreads), smem, stream, a, lpc, nchunk);
}
}  // namespace

bool scan_takes_dt(int seq_len, int states) { return seq_len <= 4 && states <= 128; }

template <typename T>
int launch_selective_scan(const ScanArgs<T>& a, cudaStream_t stream)
{
    if (a.g.rows() == 0) return TLLM_OK;
    if (a.states < 1 || a.states > 512 || a.channels < 1) return fail(TLLM_ERR_SHAPE, "selective_scan: channels=%d states=%d (1..512)", a.channels, a.states);
    const int nchunk = time_chunks(a.g.seq_len, 2);
    if (nchunk > 1 && !a.rec) return fail(TLLM_ERR_NULL, "selective_scan: no record buffer");
    // few tokens: more lanes per channel; many: more states per lane (fewer instructions per state)
    const int ns = scan_takes_dt(a.g.seq_len, a.states) ? 4 : 16;
    if (a.dt_w && (ns != 4 || a.dt_rank % 8 || a.dt_off % 8 || a.ld_bc % 8))
        return fail(TLLM_ERR_SHAPE, "selective_scan: dt_rank=%d with %d tokens", a.dt_rank, a.g.seq_len);
    int lpc = 1;
    while (lpc * ns < a.states) lpc *= 2;
    if (ns == 4)
        return a.dt_w ? scan_passes<T, 4, 1, false, true>(a, lpc, nchunk, stream) : scan_passes<T, 4, 1, false, false>(a, lpc, nchunk, stream);
    return lpc == 1 ? scan_passes<T, 16, 8, true, false>(a, lpc, nchunk, stream) : scan_passes<T, 16, 8, false, false>(a, lpc, nchunk, stream);
}

template <typename T>
int launch_gated_scan(const GatedScanArgs<T>& a, cudaStream_t stream)
{
    if (a.g.rows() == 0) return TLLM_OK;
    if (a.channels < 1 || a.block < 1 || a.channels % a.block) return fail(TLLM_ERR_SHAPE, "gated_scan: channels=%d block=%d", a.channels, a.block);
    const int nchunk = time_chunks(a.g.seq_len, 1);
    if (nchunk > 1 && !a.rec) return fail(TLLM_ERR_NULL, "gated_scan: no record buffer");
    const unsigned gx = (a.channels + kGateThreads - 1) / kGateThreads;
    if (nchunk > 1) {
        const int st = launch_pdl("gated_scan", gated_scan_kernel<T, false>, dim3(gx, nchunk - 1, a.g.n_seq), dim3(kGateThreads), 0, stream, a, nchunk);
        if (st) return st;
    }
    return launch_pdl("gated_scan", gated_scan_kernel<T, true>, dim3(gx, nchunk, a.g.n_seq), dim3(kGateThreads), 0, stream, a, nchunk);
}

#define TLLM_INSTANTIATE(T)                                                \
    template int launch_norm_chain<T>(const NormArgs<T>&, cudaStream_t);    \
    template int launch_causal_conv<T>(const ConvArgs<T>&, cudaStream_t);   \
    template int launch_selective_scan<T>(const ScanArgs<T>&, cudaStream_t); \
    template int launch_gated_scan<T>(const GatedScanArgs<T>&, cudaStream_t);
TLLM_INSTANTIATE(bf16)
TLLM_INSTANTIATE(float)
#undef TLLM_INSTANTIATE

}  // namespace tllm
