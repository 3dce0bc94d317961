// Residual chain, causal convolution and the two recurrences of the mixed-layer decoder.
//
// All of them are bound by memory or by the length of the sequence, not by arithmetic.  A
// recurrence over many tokens is cut into time chunks inside one CTA: every chunk first runs
// from a zero state and records its final state and its total decay, the chunks' true initial
// states follow from those records, and a second pass over the chunk produces the outputs.
// A single token takes the same code with one chunk.
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
    if (a.y && a.w_post) {
        const float* y = a.y + (size_t)row * a.w;
        float ss = 0.f;
        for (int i = threadIdx.x; i < n4; i += kNormThreads) {
            const float4 v = load4(y + 4 * i);
            store4(vals + 4 * i, v);
            ss += sq4(v);
        }
        rinv = 1.0f / sqrtf(cta_sum(ss, sh) / (float)a.width + a.eps);
    }
    float ss = 0.f;
    for (int i = threadIdx.x; i < n4; i += kNormThreads) {
        float4 v;
        if (a.table) {
            v = load4(a.table + (size_t)a.tokens[row] * a.w + 4 * i);
            if (a.emb) store4(a.emb + (size_t)row * a.w + 4 * i, v);
        } else {
            v = load4(x + 4 * i);
        }
        if (a.y) {
            if (a.w_post) {
                const float4 y = load4(vals + 4 * i), w = load4(a.w_post + 4 * i);
                v.x += y.x * rinv * w.x;
                v.y += y.y * rinv * w.y;
                v.z += y.z * rinv * w.z;
                v.w += y.w * rinv * w.w;
            } else {
                const float4 y = load4(a.y + (size_t)row * a.w + 4 * i);
                v.x += y.x;
                v.y += y.y;
                v.z += y.z;
                v.w += y.w;
            }
        }
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
    }
    if (!a.w_next) return;
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
#pragma unroll 4
        for (int t = t0; t < t1; t++) {
#pragma unroll
            for (int j = 0; j + 1 < TAPS; j++) win[j] = win[j + 1];
            win[TAPS - 1] = input(t);
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
constexpr int kScanCh = 16;          // channels per CTA
constexpr int kScanMaxThreads = 512;
constexpr int kScanU = 4;            // tokens loaded together

// A channel is served by `lpc` lanes with NS states each; lane l holds states l * NS ...
template <typename T, int NS>
__global__ void __launch_bounds__(kScanMaxThreads)
selective_scan_kernel(const ScanArgs<T> a, int lpc, int nchunk)
{
    extern __shared__ __align__(16) float smem[];
    pdl_launch_dependents();
    const int per = kScanCh * lpc, chunk = threadIdx.x / per, rem = threadIdx.x - chunk * per;
    const int cl = rem / lpc, l = rem - cl * lpc;
    const int c_raw = blockIdx.x * kScanCh + cl;
    const bool live = c_raw < a.channels;
    const int c = live ? c_raw : a.channels - 1, b = blockIdx.y;
    const int n = a.g.seq_len, s0 = l * NS, st8 = (a.states + 7) & ~7;
    const int len = (n + nchunk - 1) / nchunk, t0 = min(n, chunk * len), t1 = min(n, t0 + len);
    float* sl = smem;                                          // [nchunk][kScanCh][lpc * NS] chunk states
    float* sd = smem + (size_t)nchunk * kScanCh * lpc * NS;    // [nchunk][kScanCh] sums of dt

    float A[NS], S[NS];
#pragma unroll
    for (int j = 0; j < NS; j++) {
        A[j] = (s0 + j < a.states) ? a.a2[(size_t)c * a.states + s0 + j] : 0.f;
        S[j] = 0.f;
    }
    const float D = a.d ? a.d[c] : 0.f;
    pdl_wait();
    const bool fresh = (a.g.pos_dev ? *a.g.pos_dev : a.g.start_pos) == 0;
    const size_t row0 = (size_t)b * n;
    const float* dtp = a.dt + row0 * a.channels + c;
    const T* xp = a.x + row0 * a.channels + c;
    const T* bp = a.bc + row0 * a.ld_bc + a.b_off + s0;
    const T* cp = a.bc + row0 * a.ld_bc + a.c_off + s0;
    const T* zp = a.z ? a.z + row0 * a.ld_z + c : nullptr;
    T* yp = a.y + row0 * a.channels + c;
    float* stp = a.state + (size_t)(a.g.first_slot + b) * a.slot_stride + (size_t)c * a.states;

    // tokens [t, t + kScanU) of the chunk; with_y: also the outputs.  Past the end dt = x = 0,
    // which leaves the state as it is.
    float sum_dt = 0.f;
    auto group = [&](int t, bool with_y) {
        float dt[kScanU], x[kScanU], Bv[kScanU][NS], Cv[kScanU][NS];
#pragma unroll
        for (int u = 0; u < kScanU; u++) {
            const int tt = t + u;
            const bool in = tt < t1;
            dt[u] = in ? dtp[(size_t)tt * a.channels] : 0.f;
            x[u] = in ? to_f<T>(xp[(size_t)tt * a.channels]) : 0.f;
#pragma unroll
            for (int j = 0; j < NS; j += 4) {
                float4 v = make_float4(0.f, 0.f, 0.f, 0.f), w = v;
                if (in && s0 + j < st8) {
                    v = load4(bp + (size_t)tt * a.ld_bc + j);
                    if (with_y) w = load4(cp + (size_t)tt * a.ld_bc + j);
                }
                Bv[u][j] = v.x; Bv[u][j + 1] = v.y; Bv[u][j + 2] = v.z; Bv[u][j + 3] = v.w;
                Cv[u][j] = w.x; Cv[u][j + 1] = w.y; Cv[u][j + 2] = w.z; Cv[u][j + 3] = w.w;
            }
        }
        float y[kScanU];
#pragma unroll
        for (int u = 0; u < kScanU; u++) {
            const float dx = dt[u] * x[u];
            sum_dt += dt[u];
            y[u] = 0.f;
#pragma unroll
            for (int j = 0; j < NS; j++) {
                S[j] = fmaf(exp2f(dt[u] * A[j]), S[j], dx * Bv[u][j]);
                y[u] = fmaf(S[j], Cv[u][j], y[u]);
            }
        }
        if (with_y) {
#pragma unroll
            for (int u = 0; u < kScanU; u++)
                for (int o = lpc >> 1; o > 0; o >>= 1) y[u] += __shfl_xor_sync(0xffffffffu, y[u], o);
#pragma unroll
            for (int u = 0; u < kScanU; u++) {
                const int tt = t + u;
                if (live && tt < t1 && l == u % lpc) {
                    float v = fmaf(D, x[u], y[u]);
                    if (zp) {
                        const float zz = to_f<T>(zp[(size_t)tt * a.ld_z]);
                        v *= zz * sigmoid_f(zz);
                    }
                    yp[(size_t)tt * a.channels] = from_f<T>(v);
                }
            }
        }
    };

    if (nchunk > 1) {
        for (int t = t0; t < t1; t += kScanU) group(t, false);
#pragma unroll
        for (int j = 0; j < NS; j++) sl[((size_t)chunk * kScanCh + cl) * (lpc * NS) + s0 + j] = S[j];
        if (l == 0) sd[chunk * kScanCh + cl] = sum_dt;
        __syncthreads();
    }
#pragma unroll
    for (int j = 0; j < NS; j++) S[j] = (!fresh && s0 + j < a.states) ? stp[s0 + j] : 0.f;
    for (int k = 0; k < chunk; k++) {
        const float d = sd[k * kScanCh + cl];
#pragma unroll
        for (int j = 0; j < NS; j++)
            S[j] = fmaf(exp2f(d * A[j]), S[j], sl[((size_t)k * kScanCh + cl) * (lpc * NS) + s0 + j]);
    }
    if (nchunk > 1) __syncthreads();          // every chunk has read the carried state
    for (int t = t0; t < t1; t += kScanU) group(t, true);
    if (live && t0 < n && t1 == n) {
#pragma unroll
        for (int j = 0; j < NS; j++)
            if (s0 + j < a.states) stp[s0 + j] = S[j];
    }
}

// ---------------------------------------------------------------------------
// Real-gated linear recurrence
// ---------------------------------------------------------------------------
constexpr int kGateCh = 32;          // channels per CTA = lanes of a warp; a warp is a time chunk
constexpr int kGateMaxChunks = 32;

template <typename T>
__global__ void __launch_bounds__(kGateCh * kGateMaxChunks)
gated_scan_kernel(const GatedScanArgs<T> a)
{
    __shared__ float sl[kGateMaxChunks][kGateCh], sa[kGateMaxChunks][kGateCh];
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31, chunk = threadIdx.x >> 5, nchunk = blockDim.x >> 5;
    const int c_raw = blockIdx.x * kGateCh + lane, b = blockIdx.y;
    const bool live = c_raw < a.channels;
    const int c = live ? c_raw : a.channels - 1;
    const int n = a.g.seq_len, len = (n + nchunk - 1) / nchunk, t0 = min(n, chunk * len), t1 = min(n, t0 + len);
    const float kc = -a.c * a.soft_lam[c];
    pdl_wait();
    const bool fresh = (a.g.pos_dev ? *a.g.pos_dev : a.g.start_pos) == 0;
    const size_t row0 = (size_t)b * n;
    const int blk = c / a.block, ci = c - blk * a.block;
    const float* rp = a.gates + row0 * 2 * a.channels + (size_t)blk * 2 * a.block + ci;
    const T* up = a.u + row0 * a.channels + c;
    const T* yp = a.y + row0 * a.ld_y + c;
    T* op = a.out + row0 * a.channels + c;
    float* stp = a.state + (size_t)(a.g.first_slot + b) * a.slot_stride + c;

    float S = 0.f, sum_log = 0.f;
    auto step = [&](int t) {
        const float r = rp[(size_t)t * 2 * a.channels], i = rp[(size_t)t * 2 * a.channels + a.block];
        const float log_a = kc * r;
        sum_log += log_a;
        // 1 - a^2 through expm1: no cancellation when a is close to one
        S = fmaf(expf(log_a), S, sqrtf(-expm1f(2.f * log_a)) * i * to_f<T>(up[(size_t)t * a.channels]));
    };
    if (nchunk > 1) {
#pragma unroll 4
        for (int t = t0; t < t1; t++) step(t);
        sl[chunk][lane] = S;
        sa[chunk][lane] = sum_log;
        __syncthreads();
    }
    S = fresh ? 0.f : *stp;
    for (int k = 0; k < chunk; k++) S = fmaf(expf(sa[k][lane]), S, sl[k][lane]);
    if (nchunk > 1) __syncthreads();          // every chunk has read the carried state
#pragma unroll 4
    for (int t = t0; t < t1; t++) {
        step(t);
        if (live) op[(size_t)t * a.channels] = from_f<T>(S * apply_act(a.act, to_f<T>(yp[(size_t)t * a.ld_y])));
    }
    if (live && t0 < n && t1 == n) *stp = S;
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

template <typename T>
int launch_selective_scan(const ScanArgs<T>& a, cudaStream_t stream)
{
    if (a.g.rows() == 0) return TLLM_OK;
    const int ns = a.states <= 128 ? 4 : a.states <= 256 ? 8 : 16;
    if (a.states < 1 || a.states > 512 || a.channels < 1) return fail(TLLM_ERR_SHAPE, "selective_scan: channels=%d states=%d (1..512)", a.channels, a.states);
    if (a.ld_bc % 4 || a.b_off % 4 || a.c_off % 4) return fail(TLLM_ERR_ALIGN, "selective_scan: B and C must start on multiples of 4");
    int lpc = 1;
    while (lpc * ns < a.states) lpc *= 2;
    int nchunk = kScanMaxThreads / (kScanCh * lpc);
    if (nchunk > a.g.seq_len / 16) nchunk = a.g.seq_len / 16;      // at least 16 tokens per chunk
    if (nchunk < 1) nchunk = 1;
    // records of the chunks; one chunk needs none
    const size_t smem = nchunk > 1 ? (size_t)nchunk * kScanCh * (lpc * ns + 1) * sizeof(float) : 0;
    const dim3 grid((a.channels + kScanCh - 1) / kScanCh, a.g.n_seq), block(kScanCh * lpc * nchunk);
    switch (ns) {
        case 4: return launch_pdl("selective_scan", selective_scan_kernel<T, 4>, grid, block, smem, stream, a, lpc, nchunk);
        case 8: return launch_pdl("selective_scan", selective_scan_kernel<T, 8>, grid, block, smem, stream, a, lpc, nchunk);
        default: return launch_pdl("selective_scan", selective_scan_kernel<T, 16>, grid, block, smem, stream, a, lpc, nchunk);
    }
}

template <typename T>
int launch_gated_scan(const GatedScanArgs<T>& a, cudaStream_t stream)
{
    if (a.g.rows() == 0) return TLLM_OK;
    if (a.channels < 1 || a.block < 1 || a.channels % a.block) return fail(TLLM_ERR_SHAPE, "gated_scan: channels=%d block=%d", a.channels, a.block);
    int nchunk = a.g.seq_len / 16;
    if (nchunk > kGateMaxChunks) nchunk = kGateMaxChunks;
    if (nchunk < 1) nchunk = 1;
    return launch_pdl("gated_scan", gated_scan_kernel<T>, dim3((a.channels + kGateCh - 1) / kGateCh, a.g.n_seq), dim3(kGateCh * nchunk),
                      0, stream, a);
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
