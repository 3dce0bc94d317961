// Launchers of the token-mixing operators of the mixed-layer decoder (mixers.cu,
// latent_attention.cu).  T is the activation type (BF16, or float in the exact 32-bit mode);
// residual stream, norms, recurrent states and everything that feeds them stay FP32.
#pragma once
#include "dense.cuh"

namespace tllm {

// Rows of a step: n_seq sequences of seq_len new tokens each (row = b * seq_len + t).  Sequence
// b lives in slot first_slot + b and its first new token sits at start_pos (or *pos_dev).  At
// position 0 recurrent state that an earlier sequence left in the slot is ignored.
struct StepGeo {
    int n_seq = 1, seq_len = 1, first_slot = 0, start_pos = 0;
    const int* pos_dev = nullptr;
    int rows() const { return n_seq * seq_len; }
};

// One step of the residual chain, one CTA per row:
//   x += y / rms(y) * w_post        (x += y when w_post is null; skipped when y is null)
//   tap = x                         (when tap is not null)
//   x += extra                      (when extra is not null)
//   h = x / rms(x) * w_next         (when w_next is not null)
// table / tokens not null: x = table[token] first (and emb = x when emb is not null).
// row_map not null: row i of h comes from row row_map[i] of x (x is only read).
// Widths are padded to `w` (a multiple of 8, padding zero everywhere); `width` divides the sums.
template <typename T>
struct NormArgs {
    const float* y = nullptr;
    const float* w_post = nullptr;
    float* x = nullptr;
    float* tap = nullptr;
    int tap_width = 0;
    const float* extra = nullptr;
    const float* w_next = nullptr;
    T* h = nullptr;
    const T* table = nullptr;
    const int* tokens = nullptr;
    float* emb = nullptr;
    const int* row_map = nullptr;
    int rows = 0, width = 0, w = 0;
    float eps = 0.f;
};
template <typename T>
int launch_norm_chain(const NormArgs<T>& a, cudaStream_t stream);

// y[t, c] = act(b[c] + sum_j w[c, j] x[t - taps + 1 + j, c]) per sequence; the inputs before the
// step come from `state` [slot][taps - 1][channels], which is left holding the last taps - 1.
template <typename T>
struct ConvArgs {
    const T* x = nullptr;      // [rows, ldx]
    int ldx = 0;
    const float* w = nullptr;  // [channels, taps]
    const float* bias = nullptr;
    T* state = nullptr;
    size_t slot_stride = 0;    // elements
    T* y = nullptr;            // [rows, channels]
    int channels = 0, taps = 0, act = kActNone;
    StepGeo g;
};
template <typename T>
int launch_causal_conv(const ConvArgs<T>& a, cudaStream_t stream);

// Selective scan: S[c, n] = exp(dt_c A[c, n]) S + dt_c x_c B_n; y_c = (sum_n S C_n + D_c x_c) silu(z_c)
template <typename T>
struct ScanArgs {
    const T* x = nullptr;      // [rows, channels]
    const float* dt = nullptr; // [rows, channels]
    const T* bc = nullptr;     // [rows, ld_bc]: B from column b_off, C from column c_off
    int ld_bc = 0, b_off = 0, c_off = 0;
    // instead of dt (scan_takes_dt): dt = softplus(dt_w . bc[dt_off ..] + dt_bias)
    const T* dt_w = nullptr;   // [channels, dt_rank]
    const float* dt_bias = nullptr;
    int dt_rank = 0, dt_off = 0;
    const T* z = nullptr;      // [rows, ld_z], null = no gate
    int ld_z = 0;
    const float* a2 = nullptr; // [channels, states], A / ln 2
    const float* d = nullptr;  // [channels]
    float* state = nullptr;    // [slot][channels][states]
    size_t slot_stride = 0;
    T* y = nullptr;            // [rows, channels]
    int channels = 0, states = 0;
    float* rec = nullptr;      // scan_record_floats, when the sequence is cut into time chunks
    StepGeo g;
};
// records of the time chunks of a scan over n_seq x seq_len tokens (0: one chunk, none needed)
bool scan_takes_dt(int seq_len, int states);
size_t scan_record_floats(int n_seq, int seq_len, int channels, int states);
template <typename T>
int launch_selective_scan(const ScanArgs<T>& a, cudaStream_t stream);

// Real-gated linear recurrence: log a = -c r softplus(lam), S = a S + sqrt(1 - a^2) i u,
// out = S * act(y).  Gates come per block of m channels: [rows, blocks, 2, m] = r then i.
template <typename T>
struct GatedScanArgs {
    const T* u = nullptr;          // [rows, channels]
    const float* gates = nullptr;  // [rows, 2 * channels]
    const float* soft_lam = nullptr;   // [channels], softplus(lam)
    float c = 8.f;
    const T* y = nullptr;          // [rows, ld_y]
    int ld_y = 0, act = kActGeluTanh;
    float* state = nullptr;        // [slot][channels]
    size_t slot_stride = 0;
    T* out = nullptr;              // [rows, channels]
    int channels = 0, block = 0;   // block: m (padded)
    float* rec = nullptr;          // scan_record_floats with one state
    StepGeo g;
};
template <typename T>
int launch_gated_scan(const GatedScanArgs<T>& a, cudaStream_t stream);

// ---- latent attention -------------------------------------------------------------------
// Cache row of a position: [latent: R | rotated key part: rot], both padded to multiples of 8.
template <typename T>
struct LatentArgs {
    // projections of the step's rows: [q: heads x (dim + rot) | latent: R | key part: rot]
    T* proj = nullptr;
    int ld = 0, q_off = 0, kv_off = 0;
    const T* gate = nullptr;           // output gate before its sigmoid, [row * gate_ld + head], or null
    int gate_ld = 0;
    int heads = 0, dim = 0, rot = 0, vdim = 0, rank = 0;   // padded sizes
    int rank_true = 0;                 // divides the sum of squares of the latent norm
    int rot_dims = 0, rot_true = 0;    // rotated entries; true size of the rotated part
    const float* kv_norm = nullptr;    // [R]
    float eps = 0.f;
    const float2* rope = nullptr;      // [position][rot_dims / 2] (cos, sin)
    T* cache = nullptr;                // [slot][max_seq][R + rot]
    size_t slot_stride = 0;
    int max_seq = 0;
    const float* sink = nullptr;       // [heads] or null
    float scale = 0.f;
    StepGeo g;
};
// Latent norm, rotation of the queries (in place) and of the shared key part, cache append.
// q_abs not null: the rotated query parts also go behind the absorbed ones, row
// [heads][R + rot].
template <typename T>
int launch_latent_prep(const LatentArgs<T>& a, T* q_abs, cudaStream_t stream);
// Attention in latent space (weights absorbed): q_abs [rows][heads][R + rot] against the cache,
// o_lat [rows][heads][R] = normalised sums of latents.  ws: latent_workspace_floats.
size_t latent_workspace_floats(int rows, int heads, int rank);
template <typename T>
int launch_latent_absorbed(const LatentArgs<T>& a, const T* q_abs, T* o_lat, float* ws, cudaStream_t stream);
// Attention over expanded keys and values of the whole context (one sequence): kx [context]
// [heads][dim], vx [context][heads][vdim], out [rows][heads][vdim] times the output gate.
bool latent_expanded_supported(const LatentArgs<bf16>& a);
int launch_latent_expanded(const LatentArgs<bf16>& a, const bf16* kx, const bf16* vx, bf16* out, cudaStream_t stream);

}  // namespace tllm
