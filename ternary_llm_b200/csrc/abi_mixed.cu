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

template <typename T>
int matrix_op(int delta, const void* qkv, const float* decay, const float* a, const float* b, const float* neg_a, const float* dt_bias,
              float q_scale, float* state, float* o, int heads, int kv_heads, int dim, int vdim, StepGeo g, cudaStream_t s)
{
    MatrixScanArgs<T> m;
    m.delta = delta != 0;
    m.q = static_cast<const T*>(qkv);
    m.k = m.q + kv_heads * dim;
    m.v = m.k + kv_heads * dim;
    m.ld = 2 * kv_heads * dim + heads * vdim;
    m.heads = heads;
    m.kv_heads = kv_heads;
    m.dim = dim;
    m.vdim = vdim;
    m.decay = decay;
    m.a = a;
    m.b = b;
    m.ld_ab = heads;
    m.neg_a = neg_a;
    m.dt_bias = dt_bias;
    m.q_scale = q_scale;
    m.state = state;
    m.slot_stride = (size_t)heads * vdim * dim;
    m.o = o;
    m.g = g;
    float* ws = nullptr;
    return with_records((matrix_scan_workspace(sizeof(T) == 2, m.delta, g.rows(), heads, kv_heads, dim, vdim) + 3) / 4, &ws, s, [&] {
        m.ws = ws;
        return launch_matrix_scan<T>(m, static_cast<const GatedNormArgs<T>*>(nullptr), s);
    });
}

template <typename T>
int experts_op(const void* h, const float* z, const void* gate_up, const void* down, float* y, int rows, int w, int ff, int n, int top, int act,
               cudaStream_t s)
{
    ExpertArgs<T> a;
    a.z = z;
    a.ld_z = a.experts = n;
    a.top = top;
    a.h = static_cast<const T*>(h);
    a.rows = rows;
    a.w = w;
    a.ff = ff;
    a.gate_up = static_cast<const T*>(gate_up);
    a.down = static_cast<const T*>(down);
    a.act = act;
    a.y = y;
    const bool few = rows <= 8 && gemv_routed_fits(top, ff, sizeof(T));
    const int m = expert_rows(rows, top, n), k = rows * top;
    // hidden, gathered rows, outputs; counts, choices, places, weights, groups
    const size_t es = sizeof(T), n_hidden = (size_t)(few ? k : m) * ff, n_rows = few ? 0 : (size_t)m * w;
    float* ws = nullptr;
    return with_records((n_hidden + 2 * n_rows) * es / 4 + 2 * (size_t)n + 3 * (size_t)k + 3 * (m / kGroupRows) + 64, &ws, s, [&]() -> int {
        a.hidden = reinterpret_cast<T*>(ws);
        if (few) return launch_experts_few<T>(a, s);
        a.gathered = a.hidden + n_hidden;
        T* out = a.gathered + n_rows;
        a.counts = reinterpret_cast<int*>(out + n_rows);
        a.chosen = a.counts + 2 * n;
        a.part_row = a.chosen + k;
        a.part_w = reinterpret_cast<float*>(a.part_row + k);
        a.groups = reinterpret_cast<int*>(a.part_w + k);
        a.group = a.groups + 1;
        int st = launch_experts_gather<T>(a, s);
        if (st) return st;
        LinearArgs<T> l;
        l.w = a.gate_up;
        l.ldw = w;
        l.w_rows = 2 * ff;
        l.x = a.gathered;
        l.ldx = w;
        l.y = a.hidden;
        l.ldy = ff;
        l.M = m;
        l.N = ff;
        l.K = w;
        l.act = act;
        l.glu = true;
        l.group = a.group;
        l.groups = a.groups;
        l.entries = n;
        if ((st = linear(l, s))) return st;
        LinearArgs<T> d;
        d.w = a.down;
        d.ldw = ff;
        d.w_rows = w;
        d.x = a.hidden;
        d.ldx = ff;
        d.y = out;
        d.ldy = w;
        d.M = m;
        d.N = w;
        d.K = ff;
        d.group = a.group;
        d.groups = a.groups;
        d.entries = n;
        if ((st = linear(d, s))) return st;
        if (cudaMemsetAsync(y, 0, (size_t)rows * w * sizeof(float), s) != cudaSuccess)
            return fail(TLLM_ERR_LAUNCH, "experts: %s", cudaGetErrorString(cudaGetLastError()));
        NormArgs<T> c;
        c.x = y;
        c.parts = out;
        c.part_row = a.part_row;
        c.part_w = a.part_w;
        c.top = top;
        c.rows = rows;
        c.width = c.w = w;
        return launch_norm_chain<T>(c, s);
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

int tllm_b200_grouped_attention(int bf16_, void* proj, const float* q_norm, const float* k_norm, float eps, const float* rope, int rot_dims,
                                void* kc, void* vc, void* o, int heads, int kv_heads, int dim, int vdim, int chunk, int cache_rows, int max_seq,
                                float scale, float out_scale, int n_seq, int seq_len, int start_pos, void* stream)
{
    if (!proj || !kc || !vc || !o || (!rope && rot_dims > 0)) return fail(TLLM_ERR_NULL, "grouped_attention: null pointer");
    if (!grouped_supported(heads, kv_heads, dim, vdim) || rot_dims < 0 || rot_dims % 2 || rot_dims > dim || chunk < 0 || max_seq < 1 || cache_rows < 1 ||
        start_pos + seq_len > max_seq || (cache_rows < max_seq && (chunk < 1 || cache_rows < chunk + seq_len)))
        return fail(TLLM_ERR_SHAPE, "grouped_attention: heads=%d/%d dim=%d vdim=%d rot=%d chunk=%d cache_rows=%d of %d", heads, kv_heads, dim, vdim,
                    rot_dims, chunk, cache_rows, max_seq);
    const int st = check_rows("grouped_attention", n_seq, seq_len, start_pos);
    if (st) return st;
    auto run = [&](auto tag) -> int {
        using T = decltype(tag);
        GroupedArgs<T> a;
        a.proj = static_cast<T*>(proj);
        a.k_off = heads * dim;
        a.v_off = a.k_off + kv_heads * dim;
        a.ld = a.v_off + kv_heads * vdim;
        a.heads = heads;
        a.kv_heads = kv_heads;
        a.dim = a.dim_true = dim;
        a.vdim = vdim;
        a.q_norm = q_norm;
        a.k_norm = k_norm;
        a.eps = eps;
        a.rope = reinterpret_cast<const float2*>(rope);
        a.rot_dims = rot_dims;
        a.kc = static_cast<T*>(kc);
        a.vc = static_cast<T*>(vc);
        a.k_slot = (size_t)cache_rows * kv_heads * dim;
        a.v_slot = (size_t)cache_rows * kv_heads * vdim;
        a.cache_rows = cache_rows;
        a.max_seq = max_seq;
        a.chunk = chunk;
        a.scale = scale;
        a.out_scale = out_scale;
        a.out = static_cast<T*>(o);
        a.ld_out = heads * vdim;
        a.g = geo(n_seq, seq_len, start_pos);
        float* ws = nullptr;
        return with_records(grouped_workspace_floats(heads, vdim), &ws, S(stream), [&] { return launch_grouped_attention<T>(a, ws, S(stream)); });
    };
    return bf16_ ? run(bf16()) : run(float());
}

int tllm_b200_matrix_scan(int bf16_, int delta, const void* qkv, const float* decay, const float* a, const float* b, const float* neg_a,
                          const float* dt_bias, float q_scale, float* state, float* o, int heads, int kv_heads, int dim, int vdim, int n_seq,
                          int seq_len, int start_pos, void* stream)
{
    if (!qkv || !state || !o || (delta ? !a || !b || !neg_a || !dt_bias : !decay)) return fail(TLLM_ERR_NULL, "matrix_scan: null pointer");
    if (heads < 1 || kv_heads < 1 || heads % kv_heads || dim < 8 || dim % 8 || dim > 512 || vdim < 8 || vdim % 8)
        return fail(TLLM_ERR_SHAPE, "matrix_scan: heads=%d/%d dim=%d vdim=%d", heads, kv_heads, dim, vdim);
    const int st = check_rows("matrix_scan", n_seq, seq_len, start_pos);
    if (st) return st;
    const StepGeo g = geo(n_seq, seq_len, start_pos);
    return bf16_ ? matrix_op<bf16>(delta, qkv, decay, a, b, neg_a, dt_bias, q_scale, state, o, heads, kv_heads, dim, vdim, g, S(stream))
                 : matrix_op<float>(delta, qkv, decay, a, b, neg_a, dt_bias, q_scale, state, o, heads, kv_heads, dim, vdim, g, S(stream));
}

int tllm_b200_gated_norm(int bf16_, const float* o, const float* w, const void* gate, void* out, int rows, int groups, int n, float eps,
                         float out_scale, int act, void* stream)
{
    if (!o || !w || !gate || !out) return fail(TLLM_ERR_NULL, "gated_norm: null pointer");
    if (rows < 1 || groups < 1 || n < 8 || n % 8) return fail(TLLM_ERR_SHAPE, "gated_norm: rows=%d groups=%d n=%d", rows, groups, n);
    const int st = check_device();
    if (st) return st;
    auto run = [&](auto tag) -> int {
        using T = decltype(tag);
        GatedNormArgs<T> a;
        a.o = o;
        a.w = w;
        a.gate = static_cast<const T*>(gate);
        a.ld_gate = a.ld_out = groups * n;
        a.act = act;
        a.eps = eps;
        a.out_scale = out_scale;
        a.out = static_cast<T*>(out);
        a.rows = rows;
        a.groups = groups;
        a.n = a.n_true = n;
        return launch_gated_norm<T>(a, S(stream));
    };
    return bf16_ ? run(bf16()) : run(float());
}

int tllm_b200_experts(int bf16_, const void* h, const float* z, const void* gate_up, const void* down, float* y, int rows, int width, int ff,
                      int experts, int top, int act, void* stream)
{
    if (!h || !z || !gate_up || !down || !y) return fail(TLLM_ERR_NULL, "experts: null pointer");
    if (rows < 1 || width < 8 || width % 8 || ff < 8 || ff % 8 || top < 1 || top > experts)
        return fail(TLLM_ERR_SHAPE, "experts: rows=%d width=%d ff=%d, %d of %d", rows, width, ff, top, experts);
    const int st = check_device();
    if (st) return st;
    return bf16_ ? experts_op<bf16>(h, z, gate_up, down, y, rows, width, ff, experts, top, act, S(stream))
                 : experts_op<float>(h, z, gate_up, down, y, rows, width, ff, experts, top, act, S(stream));
}

}  // extern "C"
