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
//   y = sum_s part_w[s] * parts[part_row[s]]   (when parts is not null: outputs of a token's experts)
//   x = alpha x + y / rms(y) * w_post  (alpha x + y when w_post is null; skipped when there is no y)
//   x = x / rms(x) * w_sum          (when w_sum is not null)
//   tap = x                         (when tap is not null)
//   x += extra                      (when extra is not null)
//   h = x / rms(x) * w_next         (when h is not null; h = x when w_next is null)
// table / tokens not null: x = table[token] first (and emb = x when emb is not null).
// row_map not null: row i of h comes from row row_map[i] of x (x is only read).
// Widths are padded to `w` (a multiple of 8, padding zero everywhere); `width` divides the sums.
template <typename T>
struct NormArgs {
    const float* y = nullptr;
    const T* parts = nullptr;          // [.., w]
    const int* part_row = nullptr;     // [rows, top]
    const float* part_w = nullptr;     // [rows, top]
    int top = 0;
    float alpha = 1.f;
    const float* w_post = nullptr;
    const float* w_sum = nullptr;
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

// ---- grouped-query attention --------------------------------------------------------------
// Query head h reads key/value head h / (heads / kv_heads); per-head RMS norm of queries and keys
// (optional), then rotation of the first rot_dims entries (i paired with i + rot_dims / 2).  With
// `chunk` > 0 position i sees only the positions of its own chunk (i / chunk), counted from the
// start of the sequence.  Cache row of a position: position % cache_rows, keys [kv_heads][dim]
// and values [kv_heads][vdim] apart.  out = out_scale * softmax(scale q.k) v.
template <typename T>
struct GroupedArgs {
    T* proj = nullptr;                 // rows of the step; queries, keys and values at these columns
    int ld = 0, q_off = 0, k_off = 0, v_off = 0;
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0, dim_true = 0;   // dim, vdim: padded sizes
    const float *q_norm = nullptr, *k_norm = nullptr;               // [dim] or null
    float eps = 0.f;
    const float2* rope = nullptr;      // [position][rot_dims / 2] (cos, sin)
    int rot_dims = 0;
    T *kc = nullptr, *vc = nullptr;    // [slot][cache_rows][kv_heads * dim], [..][kv_heads * vdim]
    size_t k_slot = 0, v_slot = 0;     // elements
    int cache_rows = 0, max_seq = 0, chunk = 0;
    float scale = 0.f, out_scale = 1.f;
    T* out = nullptr;                  // [rows, ld_out], heads * vdim entries
    int ld_out = 0;
    StepGeo g;
};
// cache rows that passes of up to `rows` tokens need
int grouped_cache_rows(int max_seq, int chunk, int rows);
bool grouped_supported(int heads, int kv_heads, int dim, int vdim);
size_t grouped_workspace_floats(int heads, int vdim);
// norms, rotations, cache append and attention of a step; ws: grouped_workspace_floats
// the attention of prompts on tcgen05 (grouped_prompt.cu); keys and values are in the cache
bool grouped_prompt_tcgen05_supported(const GroupedArgs<bf16>& a);
int launch_grouped_prompt_tcgen05(const GroupedArgs<bf16>& a, cudaStream_t stream);
template <typename T>
int launch_grouped_attention(const GroupedArgs<T>& a, float* ws, cudaStream_t stream);

// ---- recurrences on a matrix per head ------------------------------------------------------
// With S_t [vdim][dim] the state behind token t, o_t = S_t q_t and
//   delta: S_t = g S_(t-1) + beta (v_t - g S_(t-1) k_t) k_t', with unit-length q (times q_scale) and
//          k, g = exp(neg_a softplus(a + dt_bias)), beta = sigmoid(b);
//   else:  S_t = decay S_(t-1) + v_t k_t'.
// Head h reads query/key head h / (heads / kv_heads).  State [slot][heads][vdim][dim].
template <typename T>
struct MatrixScanArgs {
    bool delta = false;
    const T *q = nullptr, *k = nullptr, *v = nullptr;   // [rows, ld]
    int ld = 0;
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0;     // padded sizes
    const float* decay = nullptr;                        // [heads] (not delta)
    const float *a = nullptr, *b = nullptr;              // [rows, ld_ab] (delta)
    int ld_ab = 0;
    const float *neg_a = nullptr, *dt_bias = nullptr;    // [heads]
    float q_scale = 1.f;
    float* state = nullptr;
    size_t slot_stride = 0;
    float* o = nullptr;                                  // [rows, heads * vdim]
    void* ws = nullptr;                                  // matrix_scan_workspace bytes
    StepGeo g;
};
// bytes for a step of `rows` tokens in all
size_t matrix_scan_workspace(bool bf16_path, bool delta, int rows, int heads, int kv_heads, int dim, int vdim);
template <typename T>
struct GatedNormArgs;
// norm: null, or the norm that turns o into the mixer's output (o itself is scratch then)
template <typename T>
int launch_matrix_scan(const MatrixScanArgs<T>& a, const GatedNormArgs<T>* norm, cudaStream_t stream);

// out = out_scale * (o / rms(o) * w) * act(gate), the norm over groups of n entries (n_true of
// them count), `groups` per row
template <typename T>
struct GatedNormArgs {
    const float* o = nullptr;          // [rows, groups * n]
    const float* w = nullptr;          // per_group ? [n] : [groups * n]
    const T* gate = nullptr;           // [rows, ld_gate]
    int ld_gate = 0, act = kActSilu;
    float eps = 0.f, out_scale = 1.f;
    T* out = nullptr;                  // [rows, ld_out]
    int ld_out = 0;
    int rows = 0, groups = 1, n = 0, n_true = 0;
};
template <typename T>
int launch_gated_norm(const GatedNormArgs<T>& a, cudaStream_t stream);

// One new token per sequence of attention and linear attention side by side, in two launches:
// ranges of positions beside the state's step, then the merge beside the norm.
template <typename T>
int launch_heads_step(const GroupedArgs<T>& att, const MatrixScanArgs<T>& scan, const GatedNormArgs<T>& norm, float* ws, cudaStream_t stream);

// ---- mixture of experts ----------------------------------------------------------------------
// Router logits [rows, ld_z]; the `top` largest are chosen (the lower index on a tie) and weighed
// by the softmax over them.  Few rows: the experts' rows are streamed for each token.  Many: the
// tokens are gathered by expert, every expert's group padded to kGroupRows.
template <typename T>
struct ExpertArgs {
    const float* z = nullptr;
    int ld_z = 0, experts = 0, top = 0;
    const T* h = nullptr;              // [rows, w]
    int rows = 0, w = 0, ff = 0;       // padded sizes
    const T *gate_up = nullptr, *down = nullptr;   // [experts * 2 ff, w], [experts * w, ff]
    int act = kActSilu;
    T* hidden = nullptr;               // few: [rows * top, ff]
    float* y = nullptr;                // few: [rows, w]
    // many
    int* counts = nullptr;             // [2 * experts], zeroed by the launch
    int *chosen = nullptr, *part_row = nullptr;    // [rows, top]
    float* part_w = nullptr;                       // [rows, top]
    T* gathered = nullptr;             // [expert_rows, w]
    int *group = nullptr, *groups = nullptr;       // LinearArgs::group: [3 * expert_rows / kGroupRows], [1]
};
int expert_rows(int rows, int top, int experts);   // capacity of the gathered rows
template <typename T>
int launch_experts_few(const ExpertArgs<T>& a, cudaStream_t stream);
template <typename T>
int launch_experts_gather(const ExpertArgs<T>& a, cudaStream_t stream);

}  // namespace tllm
