// extern "C" entry points of the mixed-layer operators (include/tllm_b200_mixed.h): argument
// checks and dispatch to dense_gemv.cu / dense_gemm.cu / mixers.cu / latent_attention.cu.
#include "mixers.cuh"
#include "tllm_b200_mixed.h"

using namespace tllm;

namespace {
inline cudaStream_t S(void* s) { return static_cast<cudaStream_t>(s); }

int check_rows(const char* fn, int n_seq, int seq_len, int start_pos)
{
    if (n_seq < 1 || seq_len < 1 || start_pos < 0)
        return fail(TLLM_ERR_SHAPE, "%s: n_seq=%d seq_len=%d start_pos=%d", fn, n_seq, seq_len, start_pos);
    return check_device();
}

StepGeo geo(int n_seq, int seq_len, int start_pos)
{
    StepGeo g;
    g.n_seq = n_seq;
    g.seq_len = seq_len;
    g.start_pos = start_pos;
    return g;
}

template <typename T>
int dense_linear(const void* x, const void* w, const float* bias, void* y, int rows, int n, int cols, int act, int glu, cudaStream_t s)
{
    LinearArgs<T> l;
    l.w = static_cast<const T*>(w);
    l.ldw = cols;
    l.w_rows = glu ? 2 * n : n;
    l.x = static_cast<const T*>(x);
    l.ldx = cols;
    l.y = y;
    l.ldy = n;
    l.y_f32 = !glu;
    l.M = rows;
    l.N = n;
    l.K = cols;
    l.bias = bias;
    l.act = act;
    l.glu = glu != 0;
    return linear(l, s);
}

template <typename T>
int conv(const void* x, const float* w, const float* bias, void* state, void* y, int channels, int taps, int act, StepGeo g, cudaStream_t s)
{
    ConvArgs<T> a;
    a.x = static_cast<const T*>(x);
    a.ldx = channels;
    a.w = w;
    a.bias = bias;
    a.state = static_cast<T*>(state);
    a.slot_stride = (size_t)(taps - 1) * channels;
    a.y = static_cast<T*>(y);
    a.channels = channels;
    a.taps = taps;
    a.act = act;
    a.g = g;
    return launch_causal_conv<T>(a, s);
}

// Scratch of a stand-alone call: allocated in stream order for its size and freed behind it.
template <typename F>
int with_records(size_t floats, float** rec, cudaStream_t s, F&& launch)
{
    if (!floats) return launch();
    if (cudaMallocAsync(reinterpret_cast<void**>(rec), floats * sizeof(float), s) != cudaSuccess)
        return fail(TLLM_ERR_LAUNCH, "operator scratch: %s", cudaGetErrorString(cudaGetLastError()));
    const int st = launch();
    cudaFreeAsync(*rec, s);
    return st;
}

template <typename T>
int sel_scan(const void* x, const float* dt, const void* bc, const void* z, const float* a2, const float* d, float* state, void* y,
             int channels, int states, StepGeo g, cudaStream_t s)
{
    ScanArgs<T> a;
    a.x = static_cast<const T*>(x);
    a.dt = dt;
    a.bc = static_cast<const T*>(bc);
    a.c_off = pad8(states);
    a.ld_bc = 2 * a.c_off;
    a.z = static_cast<const T*>(z);
    a.ld_z = channels;
    a.a2 = a2;
    a.d = d;
    a.state = state;
    a.slot_stride = (size_t)channels * states;
    a.y = static_cast<T*>(y);
    a.channels = channels;
    a.states = states;
    a.g = g;
    return with_records(scan_record_floats(g.n_seq, g.seq_len, channels, states), &a.rec, s, [&] { return launch_selective_scan<T>(a, s); });
}

template <typename T>
int gate_scan(const void* u, const float* gates, const float* soft_lam, const void* y, float* state, void* out, int channels, int blocks,
              float decay, int act, StepGeo g, cudaStream_t s)
{
    GatedScanArgs<T> a;
    a.u = static_cast<const T*>(u);
    a.gates = gates;
    a.soft_lam = soft_lam;
    a.c = decay;
    a.y = static_cast<const T*>(y);
    a.ld_y = channels;
    a.act = act;
    a.state = state;
    a.slot_stride = channels;
    a.out = static_cast<T*>(out);
    a.channels = channels;
    a.block = channels / blocks;
    a.g = g;
    return with_records(scan_record_floats(g.n_seq, g.seq_len, channels, 1), &a.rec, s, [&] { return launch_gated_scan<T>(a, s); });
}

template <typename T>
LatentArgs<T> latent(const void* cache, const float* sink, int heads, int dim, int rot, int vdim, int rank, float scale, int max_seq, StepGeo g)
{
    LatentArgs<T> a;
    a.cache = static_cast<T*>(const_cast<void*>(cache));
    a.slot_stride = (size_t)max_seq * (rank + rot);
    a.max_seq = max_seq;
    a.sink = sink;
    a.heads = heads;
    a.dim = dim;
    a.rot = rot;
    a.vdim = vdim;
    a.rank = a.rank_true = rank;
    a.scale = scale;
    a.g = g;
    return a;
}

int latent_op(const LatentArgs<bf16>& a, const void* q, void* o, cudaStream_t s)
{
    float* ws = nullptr;
    return with_records(latent_workspace_floats(a.g.rows(), a.heads, a.rank), &ws, s, [&] {
        return launch_latent_absorbed<bf16>(a, static_cast<const bf16*>(q), static_cast<bf16*>(o), ws, s);
    });
}
}  // namespace

extern "C" {

int tllm_b200_dense_linear(int bf16_, const void* x, const void* w, const float* bias, void* y, int rows, int n, int cols, int act,
                           int glu, void* stream)
{
    if (!x || !w || !y) return fail(TLLM_ERR_NULL, "dense_linear: null pointer");
    if (rows < 1 || n < 1 || cols < 8 || cols % 8) return fail(TLLM_ERR_SHAPE, "dense_linear: rows=%d n=%d cols=%d (a multiple of 8)", rows, n, cols);
    const int st = check_device();
    if (st) return st;
    return bf16_ ? dense_linear<bf16>(x, w, bias, y, rows, n, cols, act, glu, S(stream))
                 : dense_linear<float>(x, w, bias, y, rows, n, cols, act, glu, S(stream));
}

int tllm_b200_causal_conv(int bf16_, const void* x, const float* w, const float* bias, void* state, void* y, int channels, int taps,
                          int act, int n_seq, int seq_len, int start_pos, void* stream)
{
    if (!x || !w || !y || (!state && taps > 1)) return fail(TLLM_ERR_NULL, "causal_conv: null pointer");
    if (channels < 8 || channels % 8 || taps < 1) return fail(TLLM_ERR_SHAPE, "causal_conv: channels=%d taps=%d", channels, taps);
    const int st = check_rows("causal_conv", n_seq, seq_len, start_pos);
    if (st) return st;
    const StepGeo g = geo(n_seq, seq_len, start_pos);
    return bf16_ ? conv<bf16>(x, w, bias, state, y, channels, taps, act, g, S(stream))
                 : conv<float>(x, w, bias, state, y, channels, taps, act, g, S(stream));
}

int tllm_b200_selective_scan(int bf16_, const void* x, const float* dt, const void* bc, const void* z, const float* a2, const float* d,
                             float* state, void* y, int channels, int states, int n_seq, int seq_len, int start_pos, void* stream)
{
    if (!x || !dt || !bc || !a2 || !state || !y) return fail(TLLM_ERR_NULL, "selective_scan: null pointer");
    if (channels < 8 || channels % 8 || states < 1) return fail(TLLM_ERR_SHAPE, "selective_scan: channels=%d states=%d", channels, states);
    const int st = check_rows("selective_scan", n_seq, seq_len, start_pos);
    if (st) return st;
    const StepGeo g = geo(n_seq, seq_len, start_pos);
    return bf16_ ? sel_scan<bf16>(x, dt, bc, z, a2, d, state, y, channels, states, g, S(stream))
                 : sel_scan<float>(x, dt, bc, z, a2, d, state, y, channels, states, g, S(stream));
}

int tllm_b200_gated_scan(int bf16_, const void* u, const float* gates, const float* soft_lam, const void* y, float* state, void* out,
                         int channels, int blocks, float decay, int act, int n_seq, int seq_len, int start_pos, void* stream)
{
    if (!u || !gates || !soft_lam || !y || !state || !out) return fail(TLLM_ERR_NULL, "gated_scan: null pointer");
    if (channels < 8 || blocks < 1 || channels % blocks || (channels / blocks) % 8)
        return fail(TLLM_ERR_SHAPE, "gated_scan: channels=%d blocks=%d", channels, blocks);
    const int st = check_rows("gated_scan", n_seq, seq_len, start_pos);
    if (st) return st;
    const StepGeo g = geo(n_seq, seq_len, start_pos);
    return bf16_ ? gate_scan<bf16>(u, gates, soft_lam, y, state, out, channels, blocks, decay, act, g, S(stream))
                 : gate_scan<float>(u, gates, soft_lam, y, state, out, channels, blocks, decay, act, g, S(stream));
}

int tllm_b200_latent_attention(int bf16_, const void* q, const void* cache, const float* sink, void* o, int heads, int rank, int rot,
                               float scale, int max_seq, int n_seq, int seq_len, int start_pos, void* stream)
{
    if (!q || !cache || !o) return fail(TLLM_ERR_NULL, "latent_attention: null pointer");
    if (heads < 1 || rank < 8 || rank % 8 || rot < 0 || rot % 8 || max_seq < 1 || start_pos + seq_len > max_seq)
        return fail(TLLM_ERR_SHAPE, "latent_attention: heads=%d rank=%d rot=%d max_seq=%d", heads, rank, rot, max_seq);
    const int st = check_rows("latent_attention", n_seq, seq_len, start_pos);
    if (st) return st;
    const StepGeo g = geo(n_seq, seq_len, start_pos);
    if (bf16_) return latent_op(latent<bf16>(cache, sink, heads, 8, rot, 8, rank, scale, max_seq, g), q, o, S(stream));
    return launch_latent_absorbed<float>(latent<float>(cache, sink, heads, 8, rot, 8, rank, scale, max_seq, g), static_cast<const float*>(q),
                                         static_cast<float*>(o), nullptr, S(stream));
}

int tllm_b200_latent_attention_expanded(const void* q, const void* kx, const void* vx, const void* cache, const float* sink,
                                        const void* gate, void* o, int heads, int dim, int rot, int vdim, int rank, float scale,
                                        int max_seq, int seq_len, int start_pos, void* stream)
{
    if (!q || !kx || !vx || !cache || !o) return fail(TLLM_ERR_NULL, "latent_attention_expanded: null pointer");
    if (heads < 1 || dim < 8 || dim % 8 || rot < 0 || rot % 8 || vdim < 8 || vdim % 8 || rank < 8 || rank % 8 || start_pos + seq_len > max_seq)
        return fail(TLLM_ERR_SHAPE, "latent_attention_expanded: heads=%d dim=%d rot=%d vdim=%d rank=%d", heads, dim, rot, vdim, rank);
    const int st = check_rows("latent_attention_expanded", 1, seq_len, start_pos);
    if (st) return st;
    LatentArgs<bf16> a = latent<bf16>(cache, sink, heads, dim, rot, vdim, rank, scale, max_seq, geo(1, seq_len, start_pos));
    a.proj = static_cast<bf16*>(const_cast<void*>(q));
    a.ld = heads * (dim + rot);
    a.gate = static_cast<const bf16*>(gate);
    a.gate_ld = heads;
    return launch_latent_expanded(a, static_cast<const bf16*>(kx), static_cast<const bf16*>(vx), static_cast<bf16*>(o), S(stream));
}

}  // extern "C"
