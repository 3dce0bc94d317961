// Dense (not ternary) linear operators of the mixed-layer decoder: BF16 or FP32 weights and
// activations, FP32 accumulation.  Every matrix is packed at load time so that rows start on
// 16-byte boundaries: `ld` elements per row, a multiple of 8, padding columns zero.
#pragma once
#include <climits>

#include <cuda_bf16.h>

#include "common.cuh"

namespace tllm {

using bf16 = __nv_bfloat16;

// element-wise function applied to (product + bias)
enum Act { kActNone = 0, kActGeluTanh = 1, kActSilu = 2, kActSoftplus = 3, kActSigmoid = 4, kActSoftcap = 5 };

// y[m, z, n] = post(sum_k W[z, n, k] x[m, z, k]),  z = 0..batch-1
template <typename T>
struct LinearArgs {
    const T* w = nullptr;        // [batch * w_rows, ldw]
    int ldw = 0, w_rows = 0;     // rows of one batch entry in w
    const T* x = nullptr;        // row stride ldx, entry z starts at column z * x_batch
    int ldx = 0, x_batch = 0;
    void* y = nullptr;           // T or float, row stride ldy, entry z starts at column z * y_batch
    int ldy = 0, y_batch = 0;
    bool y_f32 = false;
    int M = 0, N = 0, K = 0, batch = 1;   // K: a multiple of 8 (padded)
    const float* bias = nullptr; // [batch * N], null = none
    int act = kActNone;
    float act_param = 0.f;       // softcap: the cap
    // features [act_lo, act_hi) take the activation; features from f32_from on go to y2 as FP32
    // (row stride ldy2, feature f32_from first); all three multiples of 64
    int act_lo = 0, act_hi = INT_MAX, f32_from = INT_MAX;
    float* y2 = nullptr;
    int ldy2 = 0;
    // rows in groups with a matrix each (entries of w, w_rows apart): 128 rows from 128 i on use
    // entry group[3 i], i < *groups (both on the device); group[3 i + 1], [3 i + 2]: first of the
    // groups with this entry and their number; entries: matrices in w
    const int *group = nullptr, *groups = nullptr;
    int entries = 0;
    // glu: w holds N gate rows followed by N up rows; y = act(gate) * up
    bool glu = false;
    // rows with chosen entries (launch_dense_gemv_routed)
    struct {
        const float* z = nullptr;    // logits [M, ld_z]
        int ld_z = 0, experts = 0, top = 0;
    } route;
    const T* gate = nullptr;     // y *= sigmoid(gate[m * gate_ld + z])
    int gate_ld = 0;
};

// ---- what a GEMV of a decode step takes over from its neighbours --------------------------
// Staging: the step of the residual chain in mixers.cuh computed by every CTA instead of a launch
// of its own; the new residual goes to x_out, a different buffer than x_in, because every CTA
// reads the old one while the first writes.
struct GemvNorm {
    const float* y = nullptr;       // [M, K]; null: no norm staging, the vectors come from x
    float alpha = 1.f;
    const float* w_post = nullptr;  // null: plain add
    const float* w_sum = nullptr;   // null: the sum is not normed
    const float* x_in = nullptr;
    float* x_out = nullptr;
    const float* extra = nullptr;
    const float* w_next = nullptr;  // null: the vectors are the residual itself
    void* h_out = nullptr;          // the vectors, T [M, K], or null
    int width = 0;                  // true width (K is padded)
    float eps = 0.f;
};
// Tails, for one new token per sequence (vector m belongs to slot first_slot + m):
//   kTailConv: output rows [lo, hi) are the inputs of a causal convolution with carried inputs;
//     act(convolution) goes to out, the carried inputs move on, y is not written for these rows;
//   kTailGate: rows n and N + n of entry z are the two gates of channel z * N + n of a
//     real-gated recurrence whose input is x itself: state update and out = S act(y).
enum Tail { kTailNone = 0, kTailConv = 1, kTailGate = 2 };
template <typename T>
struct GemvTail {
    int kind = kTailNone;
    int lo = 0, hi = 0, taps = 0, act = kActNone;
    const float* w = nullptr;         // convolution [hi - lo, taps]
    const float* bias = nullptr;      // convolution bias or null
    T* carried = nullptr;             // [slot][taps - 1][hi - lo]
    const float* soft_lam = nullptr;  // recurrence
    float decay = 0.f;
    const T* y = nullptr;
    int ld_y = 0;
    float* state = nullptr;           // [slot][channels]
    size_t slot_stride = 0;
    int first_slot = 0, start_pos = 0;
    const int* pos_dev = nullptr;
    T* out = nullptr;                 // [M, ld_out]
    int ld_out = 0;
};

constexpr int kGroupRows = 128;     // rows that share an entry of a grouped product

// vectors one after the other against streamed weights; at most 8 vectors per pass
template <typename T>
int launch_dense_gemv(const LinearArgs<T>& a, cudaStream_t stream);
// at most 8 vectors
template <typename T>
int launch_dense_gemv_fused(const LinearArgs<T>& a, const GemvNorm& norm, const GemvTail<T>& tail, cudaStream_t stream);
// A row's chosen entries.  sum = false: row (m * top + s) of y is the (gated) product of row m of x
// with its s-th entry; sum = true: row m of y is the weighted sum over s of the products of entry s
// with columns s * K .. of row m of x.
template <typename T>
int launch_dense_gemv_routed(const LinearArgs<T>& a, bool sum, cudaStream_t stream);
bool gemv_routed_fits(int top, int k, size_t element);
// the tails need this many lanes per row
template <typename T>
bool gemv_tail_fits(int k, int taps);
// norm staging of up to 8 rows of this width, with two norm weights
template <typename T>
bool gemv_norm_fits(int k);
int launch_dense_gemm_tcgen05(const LinearArgs<bf16>& a, cudaStream_t stream);
int launch_dense_gemm_f32(const LinearArgs<float>& a, cudaStream_t stream);
// dispatch by the number of rows
int linear(const LinearArgs<bf16>& a, cudaStream_t stream);
int linear(const LinearArgs<float>& a, cudaStream_t stream);

// ---- load-time packing ---------------------------------------------------------------
// How a BF16 matrix is laid out with padding: row groups of `r` rows, `rs` source rows apart,
// become groups `rp` rows apart; column groups of `c` columns become `cp` wide.  dst row
// (i * rp + a), column (j * cp + b) = fn(src row (i * rs + a), column (j * c + b)); everything
// else of dst stays as it is (zero).  transpose: each row group is transposed (gc must be 1):
// dst row (i * rp + b), column a.
enum PackFn { kPackCopy = 0, kPackNegExpLog2e = 1, kPackSoftplus = 2, kPackNegExp = 3 };   // applied once at load, in double
struct PackSpec {
    int gr = 1, r = 1, rs = 1, rp = 1;
    int gc = 1, c = 1, cp = 1;
    bool transpose = false;
    int fn = kPackCopy;
};
template <typename D>
int launch_pack(const void* src, const PackSpec& p, D* dst, int ld, cudaStream_t stream);

// ---- small device helpers --------------------------------------------------------------
template <typename T> __device__ __forceinline__ float to_f(T v);
template <> __device__ __forceinline__ float to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f<bf16>(bf16 v) { return __bfloat162float(v); }
template <> __device__ __forceinline__ float to_f<half>(half v) { return __half2float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float sigmoid_f(float z) { return __fdividef(1.0f, 1.0f + expf(-z)); }

// z * sigmoid(2u) with u = sqrt(2/pi) (z + 0.044715 z^3): the same number as 0.5 z (1 + tanh(u))
__device__ __forceinline__ float gelu_tanh_f(float z) { return z * sigmoid_f(1.5957691216057308f * (z + 0.044715f * z * z * z)); }
// max(z, 0) + log(1 + e), e = exp(-|z|): log(1 + e) = 2 artanh(e / (2 + e)) as its power series,
// whose argument is at most 1/3 (the first term left out is below 2^-25 of the sum)
__device__ __forceinline__ float softplus_f(float z)
{
    const float e = expf(-fabsf(z)), s = __fdividef(e, 2.f + e), q = s * s;
    const float p = 1.f + q * (1.f / 3 + q * (1.f / 5 + q * (1.f / 7 + q * (1.f / 9 + q * (1.f / 11 + q * (1.f / 13))))));
    return fmaxf(z, 0.f) + 2.f * s * p;
}

// 2^x for x <= 0, flushed to zero below the normal range
__device__ __forceinline__ float exp2_neg(float x)
{
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
    return r;
}

// 1 - e^t for t <= 0: the power series near zero (no cancellation when the decay is close to
// one), the plain difference elsewhere
__device__ __forceinline__ float one_minus_exp(float t, float e)
{
    const float p = -t * (1.f + t * (1.f / 2) * (1.f + t * (1.f / 3) * (1.f + t * (1.f / 4) * (1.f + t * (1.f / 5) * (1.f + t * (1.f / 6))))));
    return t > -0.25f ? p : 1.f - e;
}

// e^t for t <= 0 given an approximation e: close to one, where the errors of a product of many
// decays would add up, from the series (rounded once)
__device__ __forceinline__ float decay_exp(float t, float e) { return 1.f - one_minus_exp(t, e); }

// 2^x, x <= 0; the exact 32-bit mode takes the series near zero
template <typename T> __device__ __forceinline__ float decay_exp2(float x);
template <> __device__ __forceinline__ float decay_exp2<bf16>(float x) { return exp2_neg(x); }
template <> __device__ __forceinline__ float decay_exp2<float>(float x) { return decay_exp(0.69314718055994531f * x, exp2_neg(x)); }

// the switch stays outside the loop over the elements
template <int N>
__device__ __forceinline__ void apply_act_n(int act, float (&v)[N], float param = 0.f)
{
    switch (act) {
        case kActGeluTanh:
#pragma unroll
            for (int i = 0; i < N; i++) v[i] = gelu_tanh_f(v[i]);
            break;
        case kActSilu:
#pragma unroll
            for (int i = 0; i < N; i++) v[i] = v[i] * sigmoid_f(v[i]);
            break;
        case kActSoftplus:
#pragma unroll
            for (int i = 0; i < N; i++) v[i] = softplus_f(v[i]);
            break;
        case kActSigmoid:
#pragma unroll
            for (int i = 0; i < N; i++) v[i] = sigmoid_f(v[i]);
            break;
        case kActSoftcap:
#pragma unroll
            for (int i = 0; i < N; i++) v[i] = param * tanhf(v[i] / param);
            break;
        default: break;
    }
}
__device__ __forceinline__ float apply_act(int act, float z, float param = 0.f)
{
    float v[1] = {z};
    apply_act_n<1>(act, v, param);
    return v[0];
}

// 16 bytes of T as floats
template <typename T> struct Vec16;
template <> struct Vec16<bf16> {
    static constexpr int n = 8;
    static __device__ __forceinline__ void unpack(const uint4& v, float* f)
    {
        const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int i = 0; i < 4; i++) {
            f[2 * i] = __uint_as_float(w[i] << 16);
            f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
        }
    }
};
template <> struct Vec16<float> {
    static constexpr int n = 4;
    static __device__ __forceinline__ void unpack(const uint4& v, float* f)
    {
        f[0] = __uint_as_float(v.x);
        f[1] = __uint_as_float(v.y);
        f[2] = __uint_as_float(v.z);
        f[3] = __uint_as_float(v.w);
    }
};

inline int pad8(int n) { return (n + 7) / 8 * 8; }

}  // namespace tllm
