// Streaming GEMV on dense weights (decode and very short portions of a prompt), and the
// load-time packing of dense matrices and parameters.
//
// HBM-bound: a row of W is read once for up to eight vectors, which are staged in shared
// memory.  A row is served by a power-of-two group of lanes (a whole warp for rows of 32 or
// more 16-byte pieces, fewer lanes for short rows such as the step-size projection of a
// selective scan).  Every lane streams its pieces through a ring of its own in shared memory
// (cp.async, three groups of four pieces; a lane reads back only what it copied, so no barrier
// is involved), and the ring runs across the ends of rows.  The first groups are requested
// before the wait on the previous kernel -- weights depend on nothing in the stream -- and a
// launch leaves room on the SM for the next one to do the same.
#include "dense.cuh"
#include "launch.cuh"
#include "route.cuh"

namespace tllm {

namespace {

constexpr int kWarps = 8;
constexpr int kPieces = 4, kGroups = 3;        // ring of a lane: groups of 16-byte pieces
constexpr int kNormVecs = 4;                   // float4s of the residual row per thread (norm staging)
constexpr int kNormMaxK = kNormVecs * kWarps * 32 * 4;
constexpr size_t kRingBytes = (size_t)kGroups * kPieces * kWarps * 32 * 16;

__device__ __forceinline__ void ring_copy(uint32_t dst, const void* src, bool valid)
{
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(valid ? 16 : 0) : "memory");
}

// sh: one word per warp, not used by an earlier sum that is still being read
__device__ __forceinline__ float gemv_cta_sum(float v, float* sh)
{
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) sh[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.f;
#pragma unroll
    for (int i = 0; i < kWarps; i++) t += sh[i];
    return t;
}

__device__ __forceinline__ float4 gemv_ld4(const float* p, int i) { return *(reinterpret_cast<const float4*>(p) + i); }

// One vector of the residual chain into shared memory; wp, ws, wn: the norm weights, staged before
// the wait on the previous kernel.  sh: 3 * kWarps words.
template <typename T>
__device__ __forceinline__ void stage_norm(const GemvNorm& f, int m, int K, T* xs, const float* wp, const float* ws, const float* wn, float* sh)
{
    const size_t row = (size_t)m * K;
    const int n4 = K >> 2;
    float4 y[kNormVecs], x[kNormVecs];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < kNormVecs; j++) {
        const int i = threadIdx.x + j * kWarps * 32;
        y[j] = x[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < n4) {
            y[j] = gemv_ld4(f.y + row, i);
            x[j] = gemv_ld4(f.x_in + row, i);
            if (f.extra) {
                const float4 e = gemv_ld4(f.extra + row, i);
                x[j].x += e.x;
                x[j].y += e.y;
                x[j].z += e.z;
                x[j].w += e.w;
            }
        }
        ss += (y[j].x * y[j].x + y[j].y * y[j].y) + (y[j].z * y[j].z + y[j].w * y[j].w);
    }
    float rinv = 1.f;
    if (f.w_post) rinv = 1.0f / sqrtf(gemv_cta_sum(ss, sh) / (float)f.width + f.eps);
    ss = 0.f;
#pragma unroll
    for (int j = 0; j < kNormVecs; j++) {
        const int i = threadIdx.x + j * kWarps * 32;
        if (i >= n4) continue;
        float4 w = make_float4(1.f, 1.f, 1.f, 1.f);
        if (f.w_post) w = reinterpret_cast<const float4*>(wp)[i];
        x[j].x = f.alpha * x[j].x + y[j].x * rinv * w.x;
        x[j].y = f.alpha * x[j].y + y[j].y * rinv * w.y;
        x[j].z = f.alpha * x[j].z + y[j].z * rinv * w.z;
        x[j].w = f.alpha * x[j].w + y[j].w * rinv * w.w;
        ss += (x[j].x * x[j].x + x[j].y * x[j].y) + (x[j].z * x[j].z + x[j].w * x[j].w);
    }
    const bool first = blockIdx.x == 0 && blockIdx.y == 0;
    auto scale = [&](float r, const float* w) {          // x *= r * w; the new sum of squares
        ss = 0.f;
#pragma unroll
        for (int j = 0; j < kNormVecs; j++) {
            const int i = threadIdx.x + j * kWarps * 32;
            if (i >= n4) continue;
            const float4 v = reinterpret_cast<const float4*>(w)[i];
            x[j].x = x[j].x * r * v.x;
            x[j].y = x[j].y * r * v.y;
            x[j].z = x[j].z * r * v.z;
            x[j].w = x[j].w * r * v.w;
            ss += (x[j].x * x[j].x + x[j].y * x[j].y) + (x[j].z * x[j].z + x[j].w * x[j].w);
        }
    };
    if (f.w_sum) scale(1.0f / sqrtf(gemv_cta_sum(ss, sh + kWarps) / (float)f.width + f.eps), ws);
    if (first) {
#pragma unroll
        for (int j = 0; j < kNormVecs; j++) {
            const int i = threadIdx.x + j * kWarps * 32;
            if (i < n4) reinterpret_cast<float4*>(f.x_out + row)[i] = x[j];
        }
    }
    if (f.w_next) scale(1.0f / sqrtf(gemv_cta_sum(ss, sh + 2 * kWarps) / (float)f.width + f.eps), wn);
#pragma unroll
    for (int j = 0; j < kNormVecs; j++) {
        const int i = threadIdx.x + j * kWarps * 32;
        if (i >= n4) continue;
        T d[4] = {from_f<T>(x[j].x), from_f<T>(x[j].y), from_f<T>(x[j].z), from_f<T>(x[j].w)};
#pragma unroll
        for (int e = 0; e < 4; e++) xs[4 * i + e] = d[e];
        if (first && f.h_out)
#pragma unroll
            for (int e = 0; e < 4; e++) static_cast<T*>(f.h_out)[row + 4 * i + e] = d[e];
    }
    __syncthreads();             // the next vector's sums reuse sh
}

enum Route { kRouteNone = 0, kRouteEach = 1, kRouteSum = 2 };

// ROUTE (one vector per CTA, blockIdx.y = place in y): the entries of w are chosen from the row's
// logits, so nothing is requested before the wait.
template <typename T, int MB, bool NORM, int TAIL, int ROUTE = kRouteNone>
__global__ void __launch_bounds__(kWarps * 32)
dense_gemv_kernel(const LinearArgs<T> a, const GemvNorm f, const GemvTail<T> t, int lanes_per_row, int m0)
{
    constexpr int V = Vec16<T>::n;
    extern __shared__ __align__(16) uint8_t smem_raw[];
    __shared__ float sh[3 * kWarps];
    // ring, then the vectors [MB][K], then with NORM the norm weights [K] each
    T* xs = reinterpret_cast<T*>(smem_raw + kRingBytes);
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int sub = lane / lanes_per_row, l = lane - sub * lanes_per_row, rpw = 32 / lanes_per_row;
    const int z = ROUTE ? 0 : blockIdx.y;
    const int xr = ROUTE == kRouteEach ? blockIdx.y / a.route.top : blockIdx.y;      // row of x (ROUTE)
    const int nv = a.K / V;                                  // 16-byte pieces per row
    const int stride = gridDim.x * kWarps * rpw;
    const int nb0 = (blockIdx.x * kWarps + warp) * rpw;
    const int parts = ROUTE == kRouteSum ? a.route.top : (TAIL == kTailGate || a.glu) ? 2 : 1;
    const T* wz = a.w + (size_t)z * a.w_rows * a.ldw;
    // ROUTE: weights and entries of the choice behind the vectors
    float* wgt = reinterpret_cast<float*>(xs + (size_t)(ROUTE == kRouteSum ? parts : MB) * a.K);
    int* idx = reinterpret_cast<int*>(wgt + a.route.top);

    // ring of this lane: piece u of slot s at ring[(s * kPieces + u) * threads]
    const uint4* ring = reinterpret_cast<const uint4*>(smem_raw) + threadIdx.x;
    const uint32_t ring32 = (uint32_t)__cvta_generic_to_shared(ring);
    int f_nb = nb0, f_part = 0, f_c = 0, f_slot = 0;         // what is requested next
    auto request = [&]() {
        if (f_nb < a.N) {
            const int n = f_nb + sub;
            const size_t r = n < a.N ? (ROUTE == kRouteSum ? (size_t)idx[f_part] * a.w_rows + n : (size_t)n + f_part * a.N) : 0;
            const T* row = wz + r * a.ldw;
#pragma unroll
            for (int u = 0; u < kPieces; u++) {
                const int c = f_c + u * lanes_per_row + l;
                const bool v = n < a.N && c < nv;
                ring_copy(ring32 + (uint32_t)((f_slot * kPieces + u) * kWarps * 32 * 16), v ? row + (size_t)c * V : wz, v);
            }
            f_c += kPieces * lanes_per_row;
            if (f_c >= nv) {
                f_c = 0;
                if (++f_part == parts) {
                    f_part = 0;
                    f_nb += stride;
                }
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        f_slot = f_slot == kGroups - 1 ? 0 : f_slot + 1;
    };
    if (!ROUTE) {
#pragma unroll
        for (int g = 0; g < kGroups; g++) request();
    }
    if (NORM) {
        float* wn = reinterpret_cast<float*>(xs + (size_t)MB * a.K);
        const float* w[3] = {f.w_next, f.w_post, f.w_sum};
#pragma unroll
        for (int p = 0; p < 3; p++) {
            if (!w[p]) continue;
            for (int i = threadIdx.x; i < a.K / 4; i += kWarps * 32) reinterpret_cast<float4*>(wn)[i] = gemv_ld4(w[p], i);
            wn += a.K;
        }
    }

    pdl_wait();
    const int mb = ROUTE ? 1 : min(MB, a.M - m0);
    if (ROUTE) {
        if (warp == 0) choose_experts(a.route.z + (size_t)xr * a.route.ld_z, a.route.experts, a.route.top, idx, wgt);
        const int n16 = ROUTE == kRouteSum ? parts * nv : nv;
        for (int i = (int)threadIdx.x - 32; i < n16; i += (kWarps - 1) * 32)
            if (i >= 0) reinterpret_cast<uint4*>(xs)[i] = *(reinterpret_cast<const uint4*>(a.x + (size_t)xr * a.ldx) + i);
        __syncthreads();
        if (ROUTE == kRouteEach) wz += (size_t)idx[blockIdx.y - xr * a.route.top] * a.w_rows * a.ldw;
#pragma unroll
        for (int g = 0; g < kGroups; g++) request();
    } else if (NORM) {
        const float* wn = reinterpret_cast<const float*>(xs + (size_t)MB * a.K);
        const float* wp = wn + (f.w_next ? a.K : 0);
        const float* ws = wp + (f.w_post ? a.K : 0);
        for (int m = 0; m < mb; m++) stage_norm<T>(f, m, a.K, xs + (size_t)m * a.K, wp, ws, wn, sh);
    } else {
        for (int i = threadIdx.x; i < mb * nv; i += kWarps * 32) {
            const int m = i / nv, c = i - m * nv;
            reinterpret_cast<uint4*>(xs + (size_t)m * a.K)[c] =
                *(reinterpret_cast<const uint4*>(a.x + (size_t)(m0 + m) * a.ldx + (size_t)z * a.x_batch) + c);
        }
    }
    for (int i = threadIdx.x + mb * nv; i < (ROUTE ? 0 : MB * nv); i += kWarps * 32) reinterpret_cast<uint4*>(xs)[i] = make_uint4(0, 0, 0, 0);
    const bool fresh = TAIL != kTailNone && (t.pos_dev ? *t.pos_dev : t.start_pos) == 0;
    __syncthreads();

    int slot = 0;
    // all lanes of a warp take the same number of trips (the shuffles name all of them)
    for (int nb = nb0; nb < a.N; nb += stride) {
        const int n = nb + sub;
        const bool valid = n < a.N;
        // what the tail needs of this row is requested before the row itself
        float hist[MB], tw = 0.f;
        const bool conv = TAIL == kTailConv && valid && n >= t.lo && n < t.hi;
        const int ch = TAIL == kTailConv ? n - t.lo : z * a.N + n, width = t.hi - t.lo;
        if (TAIL == kTailConv) {
            if (conv && l < t.taps) tw = t.w[(size_t)ch * t.taps + l];
#pragma unroll
            for (int m = 0; m < MB; m++)
                hist[m] = (conv && m < mb && l + 1 < t.taps && !fresh)
                              ? to_f<T>(t.carried[(size_t)(t.first_slot + m) * t.slot_stride + (size_t)l * width + ch]) : 0.f;
        } else if (TAIL == kTailGate) {
#pragma unroll
            for (int m = 0; m < MB; m++)
                hist[m] = (valid && m < mb && !fresh) ? t.state[(size_t)(t.first_slot + m) * t.slot_stride + ch] : 0.f;
            if (valid) tw = -t.decay * t.soft_lam[ch];
        }
        float res[2][MB];
#pragma unroll
        for (int m = 0; m < MB; m++) res[1][m] = 0.f;
        for (int part = 0; part < parts; part++) {
            float acc[MB];
#pragma unroll
            for (int m = 0; m < MB; m++) acc[m] = 0.f;
            for (int cb = l; cb - l < nv; cb += kPieces * lanes_per_row) {
                asm volatile("cp.async.wait_group %0;" ::"n"(kGroups - 1) : "memory");
                const uint4* rs = ring + slot * kPieces * kWarps * 32;
#pragma unroll
                for (int u = 0; u < kPieces; u++) {
                    const int c = min(cb + u * lanes_per_row, nv - 1);     // pieces past the row are zero
                    float wf[V];
                    Vec16<T>::unpack(rs[u * kWarps * 32], wf);
#pragma unroll
                    for (int m = 0; m < MB; m++) {
                        float xf[V];
                        Vec16<T>::unpack(*(reinterpret_cast<const uint4*>(xs + (size_t)(ROUTE == kRouteSum ? part : m) * a.K) + c), xf);
#pragma unroll
                        for (int j = 0; j < V; j++) acc[m] = fmaf(wf[j], xf[j], acc[m]);
                    }
                }
                request();
                slot = slot == kGroups - 1 ? 0 : slot + 1;
            }
            if (ROUTE == kRouteSum) {                            // the lanes' parts meet at the end
                res[0][0] = part == 0 ? wgt[0] * acc[0] : fmaf(wgt[part], acc[0], res[0][0]);
                if (part + 1 < parts) continue;
                acc[0] = res[0][0];
            }
#pragma unroll
            for (int m = 0; m < MB; m++) {
                for (int o = lanes_per_row >> 1; o > 0; o >>= 1) acc[m] += __shfl_xor_sync(0xffffffffu, acc[m], o);
                if (part == 0 || ROUTE == kRouteSum) res[0][m] = acc[m];
                else res[1][m] = acc[m];
            }
        }
        if (TAIL == kTailConv) {
            // every lane of the group holds the row's new input; lane j weighs carried input j,
            // lane taps - 1 the new one
#pragma unroll
            for (int m = 0; m < MB; m++) {
                const float v = to_f<T>(from_f<T>(res[0][m] + ((a.bias && valid) ? a.bias[n] : 0.f)));
                float s = 0.f;
                if (conv && m < mb) s = l + 1 < t.taps ? tw * hist[m] : l + 1 == t.taps ? tw * v : 0.f;
                for (int o = lanes_per_row >> 1; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
                if (conv && m < mb) {
                    T* cr = t.carried + (size_t)(t.first_slot + m) * t.slot_stride + ch;
                    if (l > 0 && l + 1 < t.taps) cr[(size_t)(l - 1) * width] = from_f<T>(hist[m]);
                    if (l + 1 == t.taps && t.taps > 1) cr[(size_t)(t.taps - 2) * width] = from_f<T>(v);
                    if (l == 0) t.out[(size_t)m * t.ld_out + ch] = from_f<T>(apply_act(t.act, s + (t.bias ? t.bias[ch] : 0.f)));
                }
            }
            if (conv) continue;
        }
        if (!valid) continue;
#pragma unroll
        for (int m = 0; m < MB; m++) {
            if (m >= mb || l != m % lanes_per_row) continue;     // one lane of the group per vector
            if (TAIL == kTailGate) {
                const float* b = a.bias + (size_t)z * 2 * a.N;
                const float r = sigmoid_f(res[0][m] + b[n]), i = sigmoid_f(res[1][m] + b[a.N + n]);
                const float log_a = tw * r, A = decay_exp(log_a, expf(log_a));
                const float S = fmaf(A, hist[m], sqrtf(one_minus_exp(2.f * log_a, A * A)) * i * to_f<T>(xs[(size_t)m * a.K + n]));
                t.state[(size_t)(t.first_slot + m) * t.slot_stride + ch] = S;
                t.out[(size_t)m * t.ld_out + ch] = from_f<T>(S * apply_act(t.act, to_f<T>(t.y[(size_t)m * t.ld_y + ch])));
                continue;
            }
            float v = res[0][m];
            if (a.bias) v += a.bias[(size_t)z * a.N + n];
            if (n >= a.f32_from) {
                a.y2[(size_t)(m0 + m) * a.ldy2 + n - a.f32_from] = v;
                continue;
            }
            if (n >= a.act_lo && n < a.act_hi) v = apply_act(a.act, v, a.act_param);
            if (a.glu) v *= res[1][m];
            if (a.gate) v *= sigmoid_f(to_f<T>(a.gate[(size_t)(m0 + m) * a.gate_ld + z]));
            const size_t o = (size_t)(ROUTE ? (int)blockIdx.y : m0 + m) * a.ldy + (size_t)z * a.y_batch + n;
            if (a.y_f32) static_cast<float*>(a.y)[o] = v;
            else static_cast<T*>(a.y)[o] = from_f<T>(v);
        }
    }
}

template <typename T>
int row_lanes(int k)
{
    const int nv = k / Vec16<T>::n;
    int lpr = 1;
    while (lpr < 32 && lpr < nv) lpr *= 2;
    return lpr;
}

constexpr size_t kSmemLimit = 220 * 1024;

template <typename T, int MB, bool NORM, int TAIL>
int launch_mb(const LinearArgs<T>& a, const GemvNorm& f, const GemvTail<T>& t, int m0, cudaStream_t stream)
{
    static bool attr[64] = {};
    static int sms[64] = {};
    int dev = 0;
    cudaGetDevice(&dev);
    if (!attr[dev]) {
        cudaFuncSetAttribute(dense_gemv_kernel<T, MB, NORM, TAIL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSmemLimit);
        cudaDeviceGetAttribute(&sms[dev], cudaDevAttrMultiProcessorCount, dev);
        attr[dev] = true;
    }
    const int lpr = row_lanes<T>(a.K);
    const int rows_per_cta = kWarps * (32 / lpr);
    int grid = (a.N + rows_per_cta - 1) / rows_per_cta;
    // two CTAs per SM: the next launch finds room and requests its weights early
    const int cap = (2 * sms[dev] + a.batch - 1) / a.batch;
    if (grid > cap) grid = cap;
    const int norms = NORM ? (f.w_next != nullptr) + (f.w_post != nullptr) + (f.w_sum != nullptr) : 0;
    const size_t smem = kRingBytes + (size_t)MB * a.K * sizeof(T) + (size_t)norms * a.K * sizeof(float);
    if (smem > kSmemLimit || (NORM && a.K > kNormMaxK)) return fail(TLLM_ERR_SHAPE, "dense_gemv: %d vectors of %d", MB, a.K);
    return launch_pdl("dense_gemv", dense_gemv_kernel<T, MB, NORM, TAIL>, dim3(grid, a.batch), dim3(kWarps * 32), smem, stream, a, f, t, lpr, m0);
}

size_t routed_smem(int top, int k, size_t element, bool sum) { return kRingBytes + (size_t)(sum ? top : 1) * k * element + (size_t)top * 8; }

template <typename T, int ROUTE>
int launch_routed(const LinearArgs<T>& a, cudaStream_t stream)
{
    static bool attr[64] = {};
    static int sms[64] = {};
    int dev = 0;
    cudaGetDevice(&dev);
    const auto kernel = dense_gemv_kernel<T, 1, false, kTailNone, ROUTE>;
    if (!attr[dev]) {
        cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSmemLimit);
        cudaDeviceGetAttribute(&sms[dev], cudaDevAttrMultiProcessorCount, dev);
        attr[dev] = true;
    }
    const size_t smem = routed_smem(a.route.top, a.K, sizeof(T), ROUTE == kRouteSum);
    if (smem > kSmemLimit) return fail(TLLM_ERR_SHAPE, "dense_gemv: %d entries of K=%d do not fit shared memory", a.route.top, a.K);
    const int lpr = row_lanes<T>(a.K), rows_per_cta = kWarps * (32 / lpr), ny = ROUTE == kRouteSum ? a.M : a.M * a.route.top;
    int grid = (a.N + rows_per_cta - 1) / rows_per_cta;
    const int cap = (2 * sms[dev] + ny - 1) / ny;
    if (grid > cap) grid = cap;
    return launch_pdl("dense_gemv_routed", kernel, dim3(grid, ny), dim3(kWarps * 32), smem, stream, a, GemvNorm(), GemvTail<T>(), lpr, 0);
}

template <typename T, bool NORM, int TAIL>
int launch_any(const LinearArgs<T>& a, const GemvNorm& f, const GemvTail<T>& t, int mb, int m0, cudaStream_t stream)
{
    switch (mb) {
        case 8: return launch_mb<T, 8, NORM, TAIL>(a, f, t, m0, stream);
        case 4: return launch_mb<T, 4, NORM, TAIL>(a, f, t, m0, stream);
        case 2: return launch_mb<T, 2, NORM, TAIL>(a, f, t, m0, stream);
        default: return launch_mb<T, 1, NORM, TAIL>(a, f, t, m0, stream);
    }
}

template <typename T>
int check_gemv(const LinearArgs<T>& a)
{
    if (a.K < 8 || a.K % 8 || a.ldw % 8 || a.ldx % 8 || a.x_batch % 8)
        return fail(TLLM_ERR_SHAPE, "dense_gemv: K=%d ldw=%d ldx=%d x_batch=%d must be multiples of 8", a.K, a.ldw, a.ldx, a.x_batch);
    if ((size_t)a.K * sizeof(T) > kSmemLimit - kRingBytes)
        return fail(TLLM_ERR_SHAPE, "dense_gemv: K=%d exceeds %d", a.K, (int)((kSmemLimit - kRingBytes) / sizeof(T)));
    return TLLM_OK;
}

}  // namespace

template <typename T>
bool gemv_tail_fits(int k, int taps)
{
    return row_lanes<T>(k) >= taps;
}
template <typename T>
bool gemv_norm_fits(int k)
{
    return k <= kNormMaxK && kRingBytes + (size_t)k * (8 * sizeof(T) + 2 * sizeof(float)) <= kSmemLimit;
}
template bool gemv_norm_fits<bf16>(int);
template bool gemv_norm_fits<float>(int);
template bool gemv_tail_fits<bf16>(int, int);
template bool gemv_tail_fits<float>(int, int);

template <typename T>
int launch_dense_gemv_fused(const LinearArgs<T>& a, const GemvNorm& f, const GemvTail<T>& t, cudaStream_t stream)
{
    if (a.M == 0 || a.N == 0 || a.batch == 0) return TLLM_OK;
    const int st = check_gemv(a);
    if (st) return st;
    if (a.M > 8 || (f.y && (a.batch != 1 || f.x_in == f.x_out))) return fail(TLLM_ERR_SHAPE, "dense_gemv (fused): %d vectors", a.M);
    if (t.kind == kTailConv && !gemv_tail_fits<T>(a.K, t.taps)) return fail(TLLM_ERR_SHAPE, "dense_gemv (fused): %d taps for K=%d", t.taps, a.K);
    const int mb = a.M >= 5 ? 8 : a.M >= 3 ? 4 : a.M;
    if (f.y)
        return t.kind == kTailConv ? launch_any<T, true, kTailConv>(a, f, t, mb, 0, stream) : launch_any<T, true, kTailNone>(a, f, t, mb, 0, stream);
    if (t.kind == kTailConv) return launch_any<T, false, kTailConv>(a, f, t, mb, 0, stream);
    if (t.kind == kTailGate) return launch_any<T, false, kTailGate>(a, f, t, mb, 0, stream);
    return launch_any<T, false, kTailNone>(a, f, t, mb, 0, stream);
}
template int launch_dense_gemv_fused<bf16>(const LinearArgs<bf16>&, const GemvNorm&, const GemvTail<bf16>&, cudaStream_t);
template int launch_dense_gemv_fused<float>(const LinearArgs<float>&, const GemvNorm&, const GemvTail<float>&, cudaStream_t);

bool gemv_routed_fits(int top, int k, size_t element) { return routed_smem(top, k, element, true) <= kSmemLimit; }

template <typename T>
int launch_dense_gemv_routed(const LinearArgs<T>& a, bool sum, cudaStream_t stream)
{
    if (a.M == 0 || a.N == 0) return TLLM_OK;
    const int st = check_gemv(a);
    if (st) return st;
    return sum ? launch_routed<T, kRouteSum>(a, stream) : launch_routed<T, kRouteEach>(a, stream);
}
template int launch_dense_gemv_routed<bf16>(const LinearArgs<bf16>&, bool, cudaStream_t);
template int launch_dense_gemv_routed<float>(const LinearArgs<float>&, bool, cudaStream_t);

template <typename T>
int launch_dense_gemv(const LinearArgs<T>& a, cudaStream_t stream)
{
    if (a.M == 0 || a.N == 0 || a.batch == 0) return TLLM_OK;
    int st = check_gemv(a);
    for (int m0 = 0; !st && m0 < a.M;) {
        const int left = a.M - m0;
        int mb = left >= 5 ? 8 : left >= 3 ? 4 : left;
        while ((size_t)mb * a.K * sizeof(T) > kSmemLimit - kRingBytes) mb /= 2;
        st = launch_any<T, false, kTailNone>(a, GemvNorm(), GemvTail<T>(), mb, m0, stream);
        m0 += mb;
    }
    return st;
}
template int launch_dense_gemv<bf16>(const LinearArgs<bf16>&, cudaStream_t);
template int launch_dense_gemv<float>(const LinearArgs<float>&, cudaStream_t);

int linear(const LinearArgs<bf16>& a, cudaStream_t stream)
{
    return a.M <= 8 ? launch_dense_gemv<bf16>(a, stream) : launch_dense_gemm_tcgen05(a, stream);
}

int linear(const LinearArgs<float>& a, cudaStream_t stream)
{
    return a.M <= 8 ? launch_dense_gemv<float>(a, stream) : launch_dense_gemm_f32(a, stream);
}

// ---------------------------------------------------------------------------
// FP32 GEMM (the exact 32-bit mode): 64 x 64 tile, 16-deep slices, 4 x 4 outputs per thread
// ---------------------------------------------------------------------------
namespace {
constexpr int kTile = 64, kSlice = 16;

__global__ void __launch_bounds__(256)
dense_gemm_f32_kernel(const LinearArgs<float> a)
{
    __shared__ float xs[kSlice][kTile + 4], ws[2][kSlice][kTile + 4];
    pdl_launch_dependents();
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;      // outputs n = 4 tx.., m = 4 ty..
    const int n0 = blockIdx.x * kTile, m0 = blockIdx.y * kTile, z = blockIdx.z;
    const int parts = a.glu ? 2 : 1;
    float acc[2][4][4] = {};
    pdl_wait();
    if (a.group && m0 / kGroupRows >= *a.groups) return;
    const float* wz = a.w + (size_t)(a.group ? a.group[3 * (m0 / kGroupRows)] : z) * a.w_rows * a.ldw;
    const float* xz = a.x + (size_t)z * a.x_batch;
    const int lr = threadIdx.x >> 2, lc = (threadIdx.x & 3) * 4;  // loader: row of the tile, 4 columns
    for (int k0 = 0; k0 < a.K; k0 += kSlice) {
        __syncthreads();
        const bool kin = k0 + lc < a.K;                           // K is a multiple of 8
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (kin && m0 + lr < a.M) v = *reinterpret_cast<const float4*>(xz + (size_t)(m0 + lr) * a.ldx + k0 + lc);
        xs[lc][lr] = v.x;
        xs[lc + 1][lr] = v.y;
        xs[lc + 2][lr] = v.z;
        xs[lc + 3][lr] = v.w;
        for (int p = 0; p < parts; p++) {
            v = make_float4(0.f, 0.f, 0.f, 0.f);
            if (kin && n0 + lr < a.N) v = *reinterpret_cast<const float4*>(wz + (size_t)(n0 + lr + p * a.N) * a.ldw + k0 + lc);
            ws[p][lc][lr] = v.x;
            ws[p][lc + 1][lr] = v.y;
            ws[p][lc + 2][lr] = v.z;
            ws[p][lc + 3][lr] = v.w;
        }
        __syncthreads();
        for (int p = 0; p < parts; p++)
#pragma unroll
            for (int k = 0; k < kSlice; k++) {
                const float4 x4 = *reinterpret_cast<const float4*>(&xs[k][ty * 4]);
                const float4 w4 = *reinterpret_cast<const float4*>(&ws[p][k][tx * 4]);
                const float xf[4] = {x4.x, x4.y, x4.z, x4.w}, wf[4] = {w4.x, w4.y, w4.z, w4.w};
#pragma unroll
                for (int i = 0; i < 4; i++)
#pragma unroll
                    for (int j = 0; j < 4; j++)
                        if (p == 0) acc[0][i][j] = fmaf(xf[i], wf[j], acc[0][i][j]);
                        else acc[1][i][j] = fmaf(xf[i], wf[j], acc[1][i][j]);
            }
    }
    float* y = static_cast<float*>(a.y);
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
            if (m >= a.M || n >= a.N) continue;
            float v = acc[0][i][j];
            if (a.bias) v += a.bias[(size_t)z * a.N + n];
            if (n >= a.f32_from) {
                a.y2[(size_t)m * a.ldy2 + n - a.f32_from] = v;
                continue;
            }
            if (n >= a.act_lo && n < a.act_hi) v = apply_act(a.act, v, a.act_param);
            if (a.glu) v *= acc[1][i][j];
            if (a.gate) v *= sigmoid_f(a.gate[(size_t)m * a.gate_ld + z]);
            y[(size_t)m * a.ldy + (size_t)z * a.y_batch + n] = v;
        }
}
}  // namespace

int launch_dense_gemm_f32(const LinearArgs<float>& a, cudaStream_t stream)
{
    if (a.M == 0 || a.N == 0 || a.batch == 0) return TLLM_OK;
    if (a.K % 8 || a.ldw % 8 || a.ldx % 8 || a.x_batch % 8)
        return fail(TLLM_ERR_SHAPE, "dense_gemm_f32: K=%d ldw=%d ldx=%d must be multiples of 8", a.K, a.ldw, a.ldx);
    return launch_pdl("dense_gemm_f32", dense_gemm_f32_kernel,
                      dim3((a.N + kTile - 1) / kTile, (a.M + kTile - 1) / kTile, a.batch), dim3(256), 0, stream, a);
}

// ---------------------------------------------------------------------------
// Load-time packing
// ---------------------------------------------------------------------------
namespace {
__device__ __forceinline__ float pack_fn(float v, int fn)
{
    const double d = (double)v;
    if (fn == kPackNegExpLog2e) return (float)(-exp(d) * 1.4426950408889634074);
    if (fn == kPackNegExp) return (float)-exp(d);
    if (fn == kPackSoftplus) return (float)(fmax(d, 0.0) + log1p(exp(-fabs(d))));
    return v;
}

template <typename D>
__global__ void __launch_bounds__(256)
pack_kernel(const bf16* __restrict__ src, const PackSpec p, D* __restrict__ dst, int ld)
{
    const size_t cols = (size_t)p.gc * p.c, total = (size_t)p.gr * p.r * cols;
    for (size_t i = (size_t)blockIdx.x * 256 + threadIdx.x; i < total; i += (size_t)gridDim.x * 256) {
        const int row = (int)(i / cols), col = (int)(i % cols);
        const int g = row / p.r, ri = row - g * p.r, h = col / p.c, ci = col - h * p.c;
        const float v = pack_fn(__bfloat162float(src[((size_t)g * p.rs + ri) * cols + col]), p.fn);
        const size_t o = p.transpose ? ((size_t)g * p.rp + ci) * ld + ri : ((size_t)g * p.rp + ri) * ld + (size_t)h * p.cp + ci;
        dst[o] = from_f<D>(v);
    }
}
}  // namespace

template <typename D>
int launch_pack(const void* src, const PackSpec& p, D* dst, int ld, cudaStream_t stream)
{
    if (!src || !dst) return fail(TLLM_ERR_NULL, "pack: null pointer");
    const bool bad = p.gr < 1 || p.r < 1 || p.rs < p.r || p.gc < 1 || p.c < 1 ||
                     (p.transpose ? (p.gc != 1 || p.rp < p.c || ld < p.r) : (p.rp < p.r || p.cp < p.c || ld < (p.gc - 1) * p.cp + p.c));
    if (bad)
        return fail(TLLM_ERR_SHAPE, "pack: rows %d x %d (%d apart) -> %d, columns %d x %d -> %d, into rows of %d", p.gr, p.r, p.rs, p.rp,
                    p.gc, p.c, p.cp, ld);
    const size_t total = (size_t)p.gr * p.r * p.gc * p.c;
    const unsigned grid = (unsigned)((total + 255) / 256 < 65536 ? (total + 255) / 256 : 65536);
    pack_kernel<D><<<grid, 256, 0, stream>>>(static_cast<const bf16*>(src), p, dst, ld);
    return check_launch("pack");
}
template int launch_pack<bf16>(const void*, const PackSpec&, bf16*, int, cudaStream_t);
template int launch_pack<float>(const void*, const PackSpec&, float*, int, cudaStream_t);

}  // namespace tllm
