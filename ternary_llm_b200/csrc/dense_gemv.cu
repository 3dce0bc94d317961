// Streaming GEMV on dense weights (decode and very short portions of a prompt), and the
// load-time packing of dense matrices and parameters.
//
// HBM-bound: a row of W is read once for up to eight vectors, which are staged in shared
// memory.  A row is served by a power-of-two group of lanes (a whole warp for rows of 32 or
// more 16-byte pieces, fewer lanes for short rows such as the step-size projection of a
// selective scan), each lane keeping eight 16-byte loads in flight.  The first loads are
// issued before the wait on the previous kernel: weights depend on nothing in the stream.
#include "dense.cuh"
#include "launch.cuh"

namespace tllm {

namespace {

constexpr int kWarps = 8;
constexpr int kAhead = 8;      // 16-byte loads in flight per lane

template <typename T, int MB>
__global__ void __launch_bounds__(kWarps * 32)
dense_gemv_kernel(const LinearArgs<T> a, int lanes_per_row, int m0)
{
    constexpr int V = Vec16<T>::n;
    extern __shared__ __align__(16) uint8_t smem_raw[];
    T* xs = reinterpret_cast<T*>(smem_raw);                  // [MB][K]
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int sub = lane / lanes_per_row, l = lane - sub * lanes_per_row, rpw = 32 / lanes_per_row;
    const int z = blockIdx.y;
    const int nv = a.K / V;                                  // 16-byte pieces per row
    const int stride = gridDim.x * kWarps * rpw;
    const int first = (blockIdx.x * kWarps + warp) * rpw + sub;
    const T* wz = a.w + (size_t)z * a.w_rows * a.ldw;

    uint4 pre[kAhead];
    auto fetch = [&](const T* row, int c0, bool valid) {
#pragma unroll
        for (int u = 0; u < kAhead; u++) {
            const int c = c0 + u * lanes_per_row;
            pre[u] = (valid && c < nv) ? __ldcs(reinterpret_cast<const uint4*>(row) + c) : make_uint4(0, 0, 0, 0);
        }
    };
    fetch(wz + (size_t)first * a.ldw, l, first < a.N);

    pdl_wait();
    const int mb = min(MB, a.M - m0);
    for (int i = threadIdx.x; i < mb * nv; i += kWarps * 32) {
        const int m = i / nv, c = i - m * nv;
        reinterpret_cast<uint4*>(xs + (size_t)m * a.K)[c] =
            *(reinterpret_cast<const uint4*>(a.x + (size_t)(m0 + m) * a.ldx + (size_t)z * a.x_batch) + c);
    }
    for (int i = threadIdx.x + mb * nv; i < MB * nv; i += kWarps * 32) reinterpret_cast<uint4*>(xs)[i] = make_uint4(0, 0, 0, 0);
    __syncthreads();

    const int parts = a.glu ? 2 : 1;
    // all lanes of a warp take the same number of trips (the shuffles name all of them)
    for (int nb = (blockIdx.x * kWarps + warp) * rpw; nb < a.N; nb += stride) {
        const int n = nb + sub;
        float res[2][MB];
        for (int part = 0; part < parts; part++) {
            const bool valid = n < a.N;
            const T* row = wz + (size_t)(valid ? n + part * a.N : 0) * a.ldw;
            float acc[MB];
#pragma unroll
            for (int m = 0; m < MB; m++) acc[m] = 0.f;
            for (int c0 = l; c0 < nv; c0 += kAhead * lanes_per_row) {
                if (!(nb == (blockIdx.x * kWarps + warp) * rpw && part == 0 && c0 == l)) fetch(row, c0, valid);
#pragma unroll
                for (int u = 0; u < kAhead; u++) {
                    const int c = min(c0 + u * lanes_per_row, nv - 1);     // pieces past the row are zero
                    float wf[V];
                    Vec16<T>::unpack(pre[u], wf);
#pragma unroll
                    for (int m = 0; m < MB; m++) {
                        float xf[V];
                        Vec16<T>::unpack(*(reinterpret_cast<const uint4*>(xs + (size_t)m * a.K) + c), xf);
#pragma unroll
                        for (int j = 0; j < V; j++) acc[m] = fmaf(wf[j], xf[j], acc[m]);
                    }
                }
            }
#pragma unroll
            for (int m = 0; m < MB; m++) {
                for (int o = lanes_per_row >> 1; o > 0; o >>= 1) acc[m] += __shfl_xor_sync(0xffffffffu, acc[m], o);
                res[part][m] = acc[m];
            }
        }
        if (n >= a.N) continue;
#pragma unroll
        for (int m = 0; m < MB; m++) {
            if (m >= mb || l != m % lanes_per_row) continue;     // one lane of the group per vector
            float v = res[0][m];
            if (a.bias) v += a.bias[(size_t)z * a.N + n];
            v = apply_act(a.act, v);
            if (a.glu) v *= res[1][m];
            if (a.gate) v *= sigmoid_f(to_f<T>(a.gate[(size_t)(m0 + m) * a.gate_ld + z]));
            const size_t o = (size_t)(m0 + m) * a.ldy + (size_t)z * a.y_batch + n;
            if (a.y_f32) static_cast<float*>(a.y)[o] = v;
            else static_cast<T*>(a.y)[o] = from_f<T>(v);
        }
    }
}

template <typename T, int MB>
int launch_mb(const LinearArgs<T>& a, int m0, cudaStream_t stream)
{
    static bool attr[64] = {};
    static int sms[64] = {};
    int dev = 0;
    cudaGetDevice(&dev);
    if (!attr[dev]) {
        cudaFuncSetAttribute(dense_gemv_kernel<T, MB>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        cudaDeviceGetAttribute(&sms[dev], cudaDevAttrMultiProcessorCount, dev);
        attr[dev] = true;
    }
    const int nv = a.K / Vec16<T>::n;
    int lpr = 1;
    while (lpr < 32 && lpr < nv) lpr *= 2;
    const int rows_per_cta = kWarps * (32 / lpr);
    int grid = (a.N + rows_per_cta - 1) / rows_per_cta;
    const int cap = sms[dev] * 8;
    if (grid > cap) grid = cap;
    return launch_pdl("dense_gemv", dense_gemv_kernel<T, MB>, dim3(grid, a.batch), dim3(kWarps * 32),
                      (size_t)MB * a.K * sizeof(T), stream, a, lpr, m0);
}

}  // namespace

template <typename T>
int launch_dense_gemv(const LinearArgs<T>& a, cudaStream_t stream)
{
    if (a.M == 0 || a.N == 0 || a.batch == 0) return TLLM_OK;
    if (a.K < 8 || a.K % 8 || a.ldw % 8 || a.ldx % 8 || a.x_batch % 8)
        return fail(TLLM_ERR_SHAPE, "dense_gemv: K=%d ldw=%d ldx=%d x_batch=%d must be multiples of 8", a.K, a.ldw, a.ldx, a.x_batch);
    const size_t limit = 200 * 1024;
    if ((size_t)a.K * sizeof(T) > limit) return fail(TLLM_ERR_SHAPE, "dense_gemv: K=%d exceeds %d", a.K, (int)(limit / sizeof(T)));
    for (int m0 = 0; m0 < a.M;) {
        const int left = a.M - m0;
        int mb = left >= 5 ? 8 : left >= 3 ? 4 : left;
        while ((size_t)mb * a.K * sizeof(T) > limit) mb /= 2;
        int st = TLLM_OK;
        switch (mb) {
            case 8: st = launch_mb<T, 8>(a, m0, stream); break;
            case 4: st = launch_mb<T, 4>(a, m0, stream); break;
            case 2: st = launch_mb<T, 2>(a, m0, stream); break;
            default: st = launch_mb<T, 1>(a, m0, stream); break;
        }
        if (st) return st;
        m0 += mb;
    }
    return TLLM_OK;
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
    const float* wz = a.w + (size_t)z * a.w_rows * a.ldw;
    const float* xz = a.x + (size_t)z * a.x_batch;
    const int parts = a.glu ? 2 : 1;
    float acc[2][4][4] = {};
    pdl_wait();
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
            v = apply_act(a.act, v);
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
