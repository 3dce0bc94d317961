// Decoder of a list of mixer layers (include/tllm_b200_mixed.h): latent attention, selective
// scan, real-gated linear recurrence, and the mixers made of heads (grouped-query attention,
// linear attention, gated delta rule; alone or two side by side), each with an optional dense or
// routed feed-forward, norms around every sublayer or behind the sum, layers that run several
// times.
//
// The residual stream, the norms, the recurrent states and what feeds them are FP32; weights and
// activations are BF16 (or FP32 in the exact mode, the same code instantiated for float).  All
// matrices are packed at creation: every dimension that is ever contracted or addressed in
// 16-byte pieces is padded to a multiple of 8 with zero weights, matrices that share their input
// are laid out as one, and parameters are turned into what the kernels use (A / ln 2,
// softplus(lam), the rotation table), in double.
//
// A step never touches the host between its launches and takes its position from device
// memory when asked to, so the shared greedy loop (decoder.cu) replays it as a CUDA graph.
#include <cmath>
#include <map>
#include <utility>
#include <vector>

#include "decoder.cuh"
#include "layer.cuh"
#include "mixers.cuh"
#include "tllm_b200_mixed.h"

namespace tllm {

namespace {

constexpr int kMaxRows = 2048;       // tokens of a prompt that go through the layers together
constexpr int kAbsorbRows = 128;     // rows of one absorbed-attention call
constexpr int kFewRows = 8;          // up to here a step is bound by reading the weights

template <typename T>
struct Mat {
    T* p = nullptr;
    int rows = 0, ld = 0;
};

// A mixer made of heads; a layer has one, or two that share the projection in front and the one
// behind.  Columns: of the layer's projection, of its FP32 part (a, b), of the input of the output
// projection.  Padded sizes unless marked.
struct HeadPart {
    int type = 0, heads = 0, kv_heads = 0, dim = 0, dim_true = 0, vdim = 0, vdim_true = 0;
    int q = 0, k = 0, v = 0, gate = 0, a = 0, b = 0, out = 0;
    float out_scale = 1.f;
    // attention
    float scale = 0.f;
    int rot_dims = 0, chunk = 0;
    const float2* rope = nullptr;
    float *q_norm = nullptr, *k_norm = nullptr;
    // linear attention, delta rule
    float *norm = nullptr, *decay = nullptr, *neg_a = nullptr, *dt_bias = nullptr, *conv = nullptr;
    int taps = 0, in_act = 0, gate_act = 0;
    int conv_channels() const { return 2 * kv_heads * dim + heads * vdim; }
};

template <typename T>
struct MixLayer {
    int type = 0;
    std::vector<HeadPart> parts;
    int in_ld = 0;                             // projected columns kept in T
    int act_lo = 0, act_hi = INT_MAX, in_act = kActNone, f32_from = INT_MAX, n_f32 = 0;
    int experts = 0, top = 0;
    Mat<T> router;
    bool few = false;                          // the experts' rows may be streamed token by token
    bool has_ff() const { return ff > 0; }
    float *norm1 = nullptr, *norm1b = nullptr, *norm2 = nullptr, *norm2b = nullptr;
    Mat<T> gate_up, down, in, out;
    int ff = 0, ff_act = 0;
    // latent attention (padded sizes)
    int heads = 0, dim = 0, rot = 0, rot_true = 0, rot_dims = 0, vdim = 0, rank = 0, rank_true = 0;
    float scale = 0.f;
    Mat<T> k_up, k_up_t, v_up;
    float *kv_norm = nullptr, *sink = nullptr;
    bool head_gate = false;
    const float2* rope = nullptr;
    // recurrences (padded sizes)
    int ch = 0, taps = 0, state = 0, st8 = 0, dt8 = 0, blocks = 0, block = 0, gate_act = 0;
    float decay = 0.f;
    Mat<T> x, dt, gates;
    float *in_bias = nullptr, *conv = nullptr, *conv_bias = nullptr, *dt_bias = nullptr, *a2 = nullptr, *d = nullptr;
    float *gate_bias = nullptr, *soft_lam = nullptr;
};

template <typename T>
struct PartState {
    T *k = nullptr, *v = nullptr, *conv = nullptr;
    float* rec = nullptr;
    size_t k_slot = 0, v_slot = 0, conv_slot = 0, rec_slot = 0;
    int cache_rows = 0;
};

// cache or state of one run of a layer, all slots
template <typename T>
struct RunState {
    PartState<T> part[2];
    T* cache = nullptr;        // latent attention
    T* conv = nullptr;
    float* rec = nullptr;
    size_t cache_slot = 0, conv_slot = 0, rec_slot = 0;     // elements per slot
};

template <typename T>
struct MixedDecoder : Decoder {
    int width = 0, w = 0;                  // w: padded
    float eps = 0.f;
    std::vector<MixLayer<T>> layers;
    std::vector<std::pair<int, bool>> order;   // (layer, add the embedding output first)
    std::vector<RunState<T>> runs;
    Mat<T> embed, out_head;
    float* final_norm = nullptr;
    bool norm_after = false;
    float alpha = 1.f, softcap = 0.f;
    bool recurrent = false, inject = false, fused_ok = true;
    int rows_cap = 0;
    std::vector<int> len;                  // tokens each slot's sequence has consumed
    std::map<std::pair<double, int>, float2*> ropes;
    // activations
    float *x = nullptr, *x2 = nullptr, *emb = nullptr, *y = nullptr, *f32buf = nullptr, *ws = nullptr, *rec = nullptr, *logits = nullptr;
    T *h = nullptr, *proj = nullptr, *mixed = nullptr, *conv_out = nullptr, *xdbc = nullptr, *q_abs = nullptr, *o_lat = nullptr;
    T *kx = nullptr, *vx = nullptr;
    float *heads_o = nullptr, *router_z = nullptr, *part_w = nullptr;
    uint8_t* scan_ws = nullptr;
    T *gathered = nullptr, *hidden = nullptr, *expert_out = nullptr;
    int *counts = nullptr, *chosen = nullptr, *part_row = nullptr, *group = nullptr, *groups = nullptr;
    int* want_dev = nullptr;
    uint8_t* backup = nullptr;
    size_t backup_bytes = 0;

    int create(const tllm_b200_mixed_desc& c, int flags, int max_batch);
    int forward(const int* tokens, int n, int start_pos, const int* pos_dev, int seq, int batch, cudaStream_t s) override;
    int forward_logits(const int* tokens, int n, int start_pos, int seq, const int* want, int n_want, float* out, float* taps,
                       cudaStream_t s) override;
    int reset(cudaStream_t) override
    {
        for (int& l : len) l = 0;
        return TLLM_OK;
    }
    void* logits_row(int seq) override { return logits + (size_t)seq * vocab; }
    int advance(int seq, int n_seq, int start_pos, int count) override;
    int save_sequence(int seq, cudaStream_t s) override { return copy_sequence(seq, true, s); }
    int restore_sequence(int seq, cudaStream_t s) override { return copy_sequence(seq, false, s); }
    int n_runs() const override { return (int)order.size(); }

private:
    int copy_sequence(int seq, bool save, cudaStream_t s);
    int mat(Mat<T>* m, int rows, int ld)
    {
        m->rows = rows;
        m->ld = ld;
        return dev_alloc(&m->p, (size_t)rows * ld, true);
    }
    int vec(float** out, const void* src, int gr, int r, int rp, int fn = kPackCopy);
    int load_layer(const tllm_b200_mixed_layer& s, MixLayer<T>& L);
    int load_heads(const tllm_b200_mixed_layer& s, MixLayer<T>& L);
    int load_part(const tllm_b200_mixed_layer& s, MixLayer<T>& L, HeadPart& p);
    int pack_rows(const void* src, int gr, int r, int rs, int rp, int gc, int c, int cp, T* dst, int ld)
    {
        PackSpec p;
        p.gr = gr; p.r = r; p.rs = rs; p.rp = rp; p.gc = gc; p.c = c; p.cp = cp;
        return launch_pack<T>(src, p, dst, ld, nullptr);
    }
    int part_state(const HeadPart& p, PartState<T>* s);
    GroupedArgs<T> grouped_args(const MixLayer<T>& L, const HeadPart& p, const PartState<T>& S, const StepGeo& g) const;
    MatrixScanArgs<T> matrix_args(const MixLayer<T>& L, const HeadPart& p, const PartState<T>& S, const StepGeo& g) const;
    GatedNormArgs<T> out_norm_args(const MixLayer<T>& L, const HeadPart& p, int n_rows) const;
    int heads_inner(const MixLayer<T>& L, const RunState<T>& R, const StepGeo& g, bool conv_done, cudaStream_t s);
    LinearArgs<T> in_product(const MixLayer<T>& L, int n_rows) const;
    LinearArgs<T> head_product(int n, float* out) const;
    int experts(const MixLayer<T>& L, int n_rows, const GemvNorm* norm, cudaStream_t s);
    bool gathers(const MixLayer<T>& L, int n_rows) const { return L.experts && (n_rows > kFewRows || !L.few); }
    int rope_table(double base, int dims, const float2** out);
    int layers_pass(const int* tokens, const StepGeo& g, float* taps, size_t tap_stride, cudaStream_t s);
    int embed_rows(const int* tokens, int rows, cudaStream_t s);
    int decode_step(const int* tokens, const StepGeo& g, float* out, cudaStream_t s);
    bool fuses(const StepGeo& g) const { return g.seq_len == 1 && g.rows() <= kFewRows && fused_ok; }
    int head(const float* rows_x, const int* row_map, int n, float* out, cudaStream_t s);
    int mixer(const MixLayer<T>& L, const RunState<T>& R, const StepGeo& g, cudaStream_t s);
    int mixer_inner(const MixLayer<T>& L, const RunState<T>& R, const StepGeo& g, cudaStream_t s);
    int attention_inner(const MixLayer<T>& L, const RunState<T>& R, const StepGeo& g, cudaStream_t s);
    ScanArgs<T> scan_args(const MixLayer<T>& L, const RunState<T>& R, const StepGeo& g) const;
    LinearArgs<T> gates_args(const MixLayer<T>& L, int n_rows) const;
    int feed_forward(const MixLayer<T>& L, int n_rows, const GemvNorm* norm, cudaStream_t s);
    bool use_expanded(const LatentArgs<T>& a) const;
    int expanded(const MixLayer<T>& L, const RunState<T>& R, const LatentArgs<T>& a, cudaStream_t s);
    LinearArgs<T> product(const Mat<T>& m, const T* in, int ldx, int k, void* out, int ldy, bool f32, int n_rows,
                          const float* bias = nullptr, int act = kActNone) const
    {
        LinearArgs<T> l;
        l.w = m.p;
        l.ldw = m.ld;
        l.w_rows = m.rows;
        l.x = in;
        l.ldx = ldx;
        l.y = out;
        l.ldy = ldy;
        l.y_f32 = f32;
        l.M = n_rows;
        l.N = m.rows;
        l.K = k;
        l.bias = bias;
        l.act = act;
        return l;
    }
    int project(const Mat<T>& m, const T* in, int ldx, int k, void* out, int ldy, bool f32, int n_rows, cudaStream_t s,
                const float* bias = nullptr, int act = kActNone)
    {
        return linear(product(m, in, ldx, k, out, ldy, f32, n_rows, bias, act), s);
    }
};

#define TRY(x_) do { if ((st = (x_)) != TLLM_OK) return st; } while (0)

// ---------------------------------------------------------------------------
// Creation
// ---------------------------------------------------------------------------
// FP32 vector of gr groups of r entries, groups rp apart
template <typename T>
int MixedDecoder<T>::vec(float** out, const void* src, int gr, int r, int rp, int fn)
{
    int st;
    TRY(dev_alloc(out, (size_t)gr * rp, true));
    PackSpec p;
    p.c = r;
    p.cp = rp;
    p.gc = gr;
    p.fn = fn;
    return launch_pack<float>(src, p, *out, gr * rp, nullptr);
}

template <typename T>
int MixedDecoder<T>::rope_table(double base, int dims, const float2** out)
{
    const auto key = std::make_pair(base, dims);
    auto it = ropes.find(key);
    if (it == ropes.end()) {
        const int half = dims / 2;
        std::vector<float2> tab((size_t)max_seq * (half > 0 ? half : 1));
        for (int i = 0; i < half; i++) {
            const double f = std::pow(base, -2.0 * i / dims);
            for (int p = 0; p < max_seq; p++) tab[(size_t)p * half + i] = make_float2((float)std::cos(p * f), (float)std::sin(p * f));
        }
        float2* d = nullptr;
        int st;
        TRY(dev_alloc(&d, tab.size(), false));
        if (cudaMemcpy(d, tab.data(), tab.size() * sizeof(float2), cudaMemcpyHostToDevice) != cudaSuccess)
            return fail(TLLM_ERR_LAUNCH, "mixed decoder: %s", cudaGetErrorString(cudaGetLastError()));
        it = ropes.emplace(key, d).first;
    }
    *out = it->second;
    return TLLM_OK;
}

template <typename T>
int MixedDecoder<T>::load_layer(const tllm_b200_mixed_layer& s, MixLayer<T>& L)
{
    int st;
    auto need = [&](std::initializer_list<int> ids) -> int {
        for (int i : ids)
            if (!s.t[i]) return fail(TLLM_ERR_NULL, "mixed decoder: tensor %d of a layer of type %d is missing", i, s.type);
        return TLLM_OK;
    };
    auto rows_to = [&](const void* src, int gr, int r, int rs, int rp, int gc, int c, int cp, T* dst, int ld) -> int {
        return pack_rows(src, gr, r, rs, rp, gc, c, cp, dst, ld);
    };
    const void* const* t = s.t;
    L.type = s.type;
    TRY(need({TLLM_T_NORM1, TLLM_T_OUT}));
    TRY(vec(&L.norm1, t[TLLM_T_NORM1], 1, width, w));
    if (s.ff > 0 && s.experts > 0) {
        TRY(need({TLLM_T_ROUTER}));
        if (s.top < 1 || s.top > s.experts) return fail(TLLM_ERR_SHAPE, "mixed decoder: %d of %d experts", s.top, s.experts);
        L.experts = s.experts;
        L.top = s.top;
        TRY(mat(&L.router, pad8(s.experts), w));
        TRY(rows_to(t[TLLM_T_ROUTER], 1, s.experts, s.experts, L.router.rows, 1, width, w, L.router.p, w));
    }
    if (t[TLLM_T_NORM1B]) TRY(vec(&L.norm1b, t[TLLM_T_NORM1B], 1, width, w));
    if (s.ff > 0) {
        TRY(need({TLLM_T_NORM2, TLLM_T_GATE, TLLM_T_UP, TLLM_T_DOWN}));
        L.ff = pad8(s.ff);
        L.ff_act = s.ff_act;
        TRY(vec(&L.norm2, t[TLLM_T_NORM2], 1, width, w));
        if (t[TLLM_T_NORM2B]) TRY(vec(&L.norm2b, t[TLLM_T_NORM2B], 1, width, w));
        const int n = L.experts ? L.experts : 1;             // matrices one behind the other
        L.few = L.experts && gemv_routed_fits(L.top, L.ff, sizeof(T));
        TRY(mat(&L.gate_up, n * 2 * L.ff, w));
        TRY(rows_to(t[TLLM_T_GATE], n, s.ff, s.ff, 2 * L.ff, 1, width, w, L.gate_up.p, w));
        TRY(rows_to(t[TLLM_T_UP], n, s.ff, s.ff, 2 * L.ff, 1, width, w, L.gate_up.p + (size_t)L.ff * w, w));
        TRY(mat(&L.down, n * w, L.ff));
        TRY(rows_to(t[TLLM_T_DOWN], n, width, width, w, 1, s.ff, L.ff, L.down.p, L.ff));
    }
    if (s.type == TLLM_MIXER_ATTENTION || s.type == TLLM_MIXER_LINEAR_ATTENTION || s.type == TLLM_MIXER_DELTA_RULE) return load_heads(s, L);
    if (s.type == TLLM_MIXER_LATENT_ATTENTION) {
        TRY(need({TLLM_T_Q, TLLM_T_KV_DOWN, TLLM_T_KV_NORM, TLLM_T_K_UP, TLLM_T_V_UP}));
        if (s.heads < 1 || s.dim < 1 || s.rot_dim < 0 || s.rot_dims < 0 || s.rot_dims > s.rot_dim || s.rot_dims % 2 || s.vdim < 1 || s.kv_rank < 1)
            return fail(TLLM_ERR_SHAPE, "mixed decoder: latent attention heads=%d dim=%d rot=%d/%d vdim=%d rank=%d", s.heads, s.dim, s.rot_dims,
                        s.rot_dim, s.vdim, s.kv_rank);
        const int H = L.heads = s.heads;
        L.dim = pad8(s.dim);
        L.rot = pad8(s.rot_dim);
        L.rot_true = s.rot_dim;
        L.rot_dims = s.rot_dims;
        L.vdim = pad8(s.vdim);
        L.rank = pad8(s.kv_rank);
        L.rank_true = s.kv_rank;
        L.scale = s.scale;
        L.head_gate = t[TLLM_T_HEAD_GATE] != nullptr;
        TRY(rope_table(s.rot_base, s.rot_dims, &L.rope));
        const int dq = L.dim + L.rot, q_rows = H * dq, kv_rows = L.rank + L.rot, g_rows = L.head_gate ? pad8(H) : 0;
        TRY(mat(&L.in, q_rows + kv_rows + g_rows, w));
        T* in = L.in.p;
        const int sq = s.dim + s.rot_dim;
        TRY(rows_to(t[TLLM_T_Q], H, s.dim, sq, dq, 1, width, w, in, w));
        if (s.rot_dim)
            TRY(rows_to(static_cast<const bf16*>(t[TLLM_T_Q]) + (size_t)s.dim * width, H, s.rot_dim, sq, dq, 1, width, w, in + (size_t)L.dim * w, w));
        in += (size_t)q_rows * w;
        TRY(rows_to(t[TLLM_T_KV_DOWN], 1, s.kv_rank, s.kv_rank, L.rank, 1, width, w, in, w));
        if (s.rot_dim)
            TRY(rows_to(static_cast<const bf16*>(t[TLLM_T_KV_DOWN]) + (size_t)s.kv_rank * width, 1, s.rot_dim, s.rot_dim, L.rot, 1, width, w,
                        in + (size_t)L.rank * w, w));
        in += (size_t)kv_rows * w;
        if (L.head_gate) TRY(rows_to(t[TLLM_T_HEAD_GATE], 1, H, H, H, 1, width, w, in, w));
        TRY(vec(&L.kv_norm, t[TLLM_T_KV_NORM], 1, s.kv_rank, L.rank));
        if (t[TLLM_T_SINK]) TRY(vec(&L.sink, t[TLLM_T_SINK], 1, H, H));
        TRY(mat(&L.k_up, H * L.dim, L.rank));
        TRY(rows_to(t[TLLM_T_K_UP], H, s.dim, s.dim, L.dim, 1, s.kv_rank, L.rank, L.k_up.p, L.rank));
        TRY(mat(&L.k_up_t, H * L.rank, L.dim));
        PackSpec p;
        p.gr = H; p.r = s.dim; p.rs = s.dim; p.rp = L.rank; p.c = s.kv_rank; p.transpose = true;
        TRY(launch_pack<T>(t[TLLM_T_K_UP], p, L.k_up_t.p, L.dim, nullptr));
        TRY(mat(&L.v_up, H * L.vdim, L.rank));
        TRY(rows_to(t[TLLM_T_V_UP], H, s.vdim, s.vdim, L.vdim, 1, s.kv_rank, L.rank, L.v_up.p, L.rank));
        TRY(mat(&L.out, w, H * L.vdim));
        TRY(rows_to(t[TLLM_T_OUT], 1, width, width, w, H, s.vdim, L.vdim, L.out.p, H * L.vdim));
    } else if (s.type == TLLM_MIXER_SELECTIVE_SCAN) {
        TRY(need({TLLM_T_IN, TLLM_T_CONV, TLLM_T_X, TLLM_T_DT, TLLM_T_A_LOG}));
        if (s.channels < 1 || s.taps < 1 || s.state < 1 || s.state > 512 || s.dt_rank < 1)
            return fail(TLLM_ERR_SHAPE, "mixed decoder: selective scan channels=%d taps=%d state=%d dt_rank=%d", s.channels, s.taps, s.state, s.dt_rank);
        recurrent = true;
        const int C = s.channels, ch = L.ch = pad8(C);
        L.taps = s.taps;
        L.state = s.state;
        L.st8 = pad8(s.state);
        L.dt8 = pad8(s.dt_rank);
        TRY(mat(&L.in, 2 * ch, w));
        TRY(rows_to(t[TLLM_T_IN], 2, C, C, ch, 1, width, w, L.in.p, w));
        TRY(mat(&L.x, L.dt8 + 2 * L.st8, ch));
        const bf16* xs = static_cast<const bf16*>(t[TLLM_T_X]);
        TRY(rows_to(xs, 1, s.dt_rank, s.dt_rank, L.dt8, 1, C, ch, L.x.p, ch));
        TRY(rows_to(xs + (size_t)s.dt_rank * C, 2, s.state, s.state, L.st8, 1, C, ch, L.x.p + (size_t)L.dt8 * ch, ch));
        TRY(mat(&L.dt, ch, L.dt8));
        TRY(rows_to(t[TLLM_T_DT], 1, C, C, ch, 1, s.dt_rank, L.dt8, L.dt.p, L.dt8));
        if (t[TLLM_T_DT_BIAS]) TRY(vec(&L.dt_bias, t[TLLM_T_DT_BIAS], 1, C, ch));
        TRY(dev_alloc(&L.a2, (size_t)ch * s.state, true));
        PackSpec p;
        p.r = p.rs = C; p.rp = ch; p.c = p.cp = s.state; p.fn = kPackNegExpLog2e;
        TRY(launch_pack<float>(t[TLLM_T_A_LOG], p, L.a2, s.state, nullptr));
        if (t[TLLM_T_D]) TRY(vec(&L.d, t[TLLM_T_D], 1, C, ch));
        TRY(mat(&L.out, w, ch));
        TRY(rows_to(t[TLLM_T_OUT], 1, width, width, w, 1, C, ch, L.out.p, ch));
    } else if (s.type == TLLM_MIXER_GATED_RECURRENCE) {
        TRY(need({TLLM_T_IN, TLLM_T_CONV, TLLM_T_Y, TLLM_T_RA, TLLM_T_RI, TLLM_T_LAM}));
        if (s.channels < 1 || s.taps < 1 || s.blocks < 1 || s.channels % s.blocks)
            return fail(TLLM_ERR_SHAPE, "mixed decoder: gated recurrence channels=%d taps=%d blocks=%d", s.channels, s.taps, s.blocks);
        recurrent = true;
        const int B = L.blocks = s.blocks, m = s.channels / B, mp = L.block = pad8(m), ch = L.ch = B * mp;
        L.taps = s.taps;
        L.decay = s.decay;
        L.gate_act = s.gate_act;
        TRY(mat(&L.in, 2 * ch, w));
        TRY(rows_to(t[TLLM_T_Y], B, m, m, mp, 1, width, w, L.in.p, w));
        TRY(rows_to(t[TLLM_T_IN], B, m, m, mp, 1, width, w, L.in.p + (size_t)ch * w, w));
        TRY(dev_alloc(&L.in_bias, (size_t)2 * ch, true));
        PackSpec p;
        p.gc = B; p.c = m; p.cp = mp;
        if (t[TLLM_T_Y_BIAS]) TRY(launch_pack<float>(t[TLLM_T_Y_BIAS], p, L.in_bias, ch, nullptr));
        if (t[TLLM_T_IN_BIAS]) TRY(launch_pack<float>(t[TLLM_T_IN_BIAS], p, L.in_bias + ch, ch, nullptr));
        TRY(mat(&L.gates, B * 2 * mp, mp));
        TRY(rows_to(t[TLLM_T_RA], B, m, m, 2 * mp, 1, m, mp, L.gates.p, mp));
        TRY(rows_to(t[TLLM_T_RI], B, m, m, 2 * mp, 1, m, mp, L.gates.p + (size_t)mp * mp, mp));
        TRY(dev_alloc(&L.gate_bias, (size_t)2 * ch, true));
        p.cp = 2 * mp;
        if (t[TLLM_T_RA_BIAS]) TRY(launch_pack<float>(t[TLLM_T_RA_BIAS], p, L.gate_bias, 2 * ch, nullptr));
        if (t[TLLM_T_RI_BIAS]) TRY(launch_pack<float>(t[TLLM_T_RI_BIAS], p, L.gate_bias + mp, 2 * ch - mp, nullptr));
        TRY(vec(&L.soft_lam, t[TLLM_T_LAM], B, m, mp, kPackSoftplus));
        TRY(mat(&L.out, w, ch));
        TRY(rows_to(t[TLLM_T_OUT], 1, width, width, w, B, m, mp, L.out.p, ch));
    } else {
        return fail(TLLM_ERR_SHAPE, "mixed decoder: unknown layer type %d", s.type);
    }
    if (L.ch) {
        const int B = L.blocks ? L.blocks : 1, m = s.channels / B, mp = L.ch / B;
        TRY(dev_alloc(&L.conv, (size_t)L.ch * L.taps, true));
        PackSpec p;
        p.gr = B; p.r = p.rs = m; p.rp = mp; p.c = p.cp = L.taps;
        TRY(launch_pack<float>(t[TLLM_T_CONV], p, L.conv, L.taps, nullptr));
        if (t[TLLM_T_CONV_BIAS]) TRY(vec(&L.conv_bias, t[TLLM_T_CONV_BIAS], B, m, mp));
    }
    return TLLM_OK;
}

// Sizes and columns are set; matrices into L.in and L.out, vectors of the mixer alone.
template <typename T>
int MixedDecoder<T>::load_part(const tllm_b200_mixed_layer& s, MixLayer<T>& L, HeadPart& p)
{
    int st;
    const void* const* t = s.t;
    auto need = [&](std::initializer_list<int> ids) -> int {
        for (int i : ids)
            if (!t[i]) return fail(TLLM_ERR_NULL, "mixed decoder: tensor %d of a mixer of type %d is missing", i, s.type);
        return TLLM_OK;
    };
    TRY(need({TLLM_T_Q, TLLM_T_K, TLLM_T_V, TLLM_T_OUT}));
    const int H = s.heads, G = s.type == TLLM_MIXER_LINEAR_ATTENTION ? H : s.kv_heads;
    auto project = [&](int slot, int heads, int n, int np, int col) -> int {
        return pack_rows(t[slot], heads, n, n, np, 1, width, w, L.in.p + (size_t)col * w, w);
    };
    const bool att = s.type == TLLM_MIXER_ATTENTION, delta = s.type == TLLM_MIXER_DELTA_RULE;
    TRY(project(TLLM_T_Q, delta ? G : H, s.dim, p.dim, p.q));
    TRY(project(TLLM_T_K, G, s.dim, p.dim, p.k));
    TRY(project(TLLM_T_V, att ? G : H, s.vdim, p.vdim, p.v));
    TRY(pack_rows(t[TLLM_T_OUT], 1, width, width, w, H, s.vdim, p.vdim, L.out.p + p.out, L.out.ld));
    if (att) {
        if (t[TLLM_T_Q_NORM]) TRY(vec(&p.q_norm, t[TLLM_T_Q_NORM], 1, s.dim, p.dim));
        if (t[TLLM_T_K_NORM]) TRY(vec(&p.k_norm, t[TLLM_T_K_NORM], 1, s.dim, p.dim));
        return rope_table(s.rot_base, s.rot_dims, &p.rope);
    }
    recurrent = true;
    TRY(need({TLLM_T_MIX_NORM, TLLM_T_MIX_GATE}));
    TRY(project(TLLM_T_MIX_GATE, H, s.vdim, p.vdim, p.gate));
    if (!delta) {
        if (!s.head_decay) return fail(TLLM_ERR_NULL, "mixed decoder: linear attention without decays");
        TRY(dev_alloc(&p.decay, (size_t)H, false));
        if (cudaMemcpy(p.decay, s.head_decay, H * sizeof(float), cudaMemcpyHostToDevice) != cudaSuccess)
            return fail(TLLM_ERR_LAUNCH, "mixed decoder: %s", cudaGetErrorString(cudaGetLastError()));
        return vec(&p.norm, t[TLLM_T_MIX_NORM], H, s.vdim, p.vdim);
    }
    TRY(need({TLLM_T_Q_CONV, TLLM_T_K_CONV, TLLM_T_V_CONV, TLLM_T_STEP, TLLM_T_DECAY, TLLM_T_DT_BIAS, TLLM_T_A_LOG}));
    TRY(project(TLLM_T_STEP, 1, H, H, L.f32_from + p.b));
    TRY(project(TLLM_T_DECAY, 1, H, H, L.f32_from + p.a));
    TRY(vec(&p.neg_a, t[TLLM_T_A_LOG], 1, H, H, kPackNegExp));
    TRY(vec(&p.dt_bias, t[TLLM_T_DT_BIAS], 1, H, H));
    TRY(vec(&p.norm, t[TLLM_T_MIX_NORM], 1, s.vdim, p.vdim));
    TRY(dev_alloc(&p.conv, (size_t)p.conv_channels() * p.taps, true));
    const int slots[3] = {TLLM_T_Q_CONV, TLLM_T_K_CONV, TLLM_T_V_CONV};
    for (int i = 0; i < 3; i++) {
        PackSpec c;
        c.gr = i < 2 ? G : H;
        c.r = c.rs = i < 2 ? s.dim : s.vdim;
        c.rp = i < 2 ? p.dim : p.vdim;
        c.c = c.cp = p.taps;
        TRY(launch_pack<float>(t[slots[i]], c, p.conv + (size_t)i * G * p.dim * p.taps, p.taps, nullptr));
    }
    return TLLM_OK;
}

// One or two mixers of heads.  Columns of the common projection: every mixer's q, k, v (and
// gate) in order, ranges that take an activation and the FP32 part on multiples of 64.
template <typename T>
int MixedDecoder<T>::load_heads(const tllm_b200_mixed_layer& s, MixLayer<T>& L)
{
    int st;
    const tllm_b200_mixed_layer* mixers[2] = {&s, s.beside};
    const int n = s.beside ? 2 : 1;
    auto pad64 = [](int v) { return (v + 63) / 64 * 64; };
    int col = 0, out = 0;
    L.parts.resize(n);
    for (int i = 0; i < n; i++) {
        const tllm_b200_mixed_layer& m = *mixers[i];
        HeadPart& p = L.parts[i];
        const bool att = m.type == TLLM_MIXER_ATTENTION, lin = m.type == TLLM_MIXER_LINEAR_ATTENTION, delta = m.type == TLLM_MIXER_DELTA_RULE;
        const int G = lin ? m.heads : m.kv_heads;
        if ((!att && !lin && !delta) || m.heads < 1 || G < 1 || m.heads % G || m.dim < 1 || m.vdim < 1 || (delta && m.taps < 1) ||
            (att && (m.rot_dims < 0 || m.rot_dims % 2 || m.rot_dims > m.dim || m.chunk < 0)))
            return fail(TLLM_ERR_SHAPE, "mixed decoder: mixer of type %d with heads=%d/%d dim=%d vdim=%d rot=%d taps=%d chunk=%d", m.type, m.heads, G,
                        m.dim, m.vdim, m.rot_dims, m.taps, m.chunk);
        if (i == 1 && !att && m.type == s.type) return fail(TLLM_ERR_SHAPE, "mixed decoder: two mixers of type %d side by side", m.type);
        p.type = m.type;
        p.heads = m.heads;
        p.kv_heads = G;
        p.dim_true = m.dim;
        p.dim = pad8(m.dim);
        p.vdim_true = m.vdim;
        p.vdim = pad8(m.vdim);
        if (att ? !grouped_supported(p.heads, G, p.dim, p.vdim) : p.dim > 512)
            return fail(TLLM_ERR_SHAPE, "mixed decoder: mixer of type %d with dim=%d vdim=%d", m.type, m.dim, m.vdim);
        p.out_scale = m.out_scale;
        p.scale = m.scale;
        p.rot_dims = m.rot_dims;
        p.chunk = m.chunk;
        p.taps = m.taps;
        p.in_act = m.in_act;
        p.gate_act = m.gate_act;
        if (lin) {
            L.act_lo = col = pad64(col);
            L.in_act = m.in_act;
        }
        p.q = col;
        p.k = p.q + (delta ? G : p.heads) * p.dim;
        p.v = p.k + G * p.dim;
        col = p.v + (att ? G : p.heads) * p.vdim;
        if (lin) L.act_hi = col = pad64(col);
        p.gate = col;
        if (!att) col += p.heads * p.vdim;
        if (delta) {
            p.b = L.n_f32;
            p.a = L.n_f32 + pad8(p.heads);
            L.n_f32 += 2 * pad8(p.heads);
        }
        p.out = out;
        out += p.heads * p.vdim;
    }
    if (L.n_f32) L.f32_from = col = pad64(col);
    L.in_ld = col;
    TRY(mat(&L.in, col + L.n_f32, w));
    TRY(mat(&L.out, w, out));
    for (int i = 0; i < n; i++) TRY(load_part(*mixers[i], L, L.parts[i]));
    return TLLM_OK;
}

// cache and state of one mixer, all slots
template <typename T>
int MixedDecoder<T>::part_state(const HeadPart& p, PartState<T>* s)
{
    int st;
    if (p.type == TLLM_MIXER_ATTENTION) {
        s->cache_rows = grouped_cache_rows(max_seq, p.chunk, rows_cap);
        if (s->cache_rows < max_seq) recurrent = true;
        s->k_slot = (size_t)s->cache_rows * p.kv_heads * p.dim;
        s->v_slot = (size_t)s->cache_rows * p.kv_heads * p.vdim;
        TRY(dev_alloc(&s->k, s->k_slot * max_batch, true));
        return dev_alloc(&s->v, s->v_slot * max_batch, true);
    }
    s->rec_slot = (size_t)p.heads * p.dim * p.vdim;
    TRY(dev_alloc(&s->rec, s->rec_slot * max_batch, true));
    if (p.type == TLLM_MIXER_DELTA_RULE && p.taps > 1) {
        s->conv_slot = (size_t)(p.taps - 1) * p.conv_channels();
        TRY(dev_alloc(&s->conv, s->conv_slot * max_batch, true));
    }
    backup_bytes += s->conv_slot * sizeof(T) + s->rec_slot * sizeof(float);
    return TLLM_OK;
}

template <typename T>
int MixedDecoder<T>::create(const tllm_b200_mixed_desc& c, int flags_, int max_batch_)
{
    int st;
    TRY(init_common(flags_, max_batch_, c.max_seq_len, c.vocab_size));
    logits_f32 = true;
    width = c.width;
    w = pad8(width);
    eps = c.norm_eps;
    len.assign(max_batch, 0);
    TRY(mat(&embed, vocab, w));
    {
        PackSpec p;
        p.r = p.rs = p.rp = vocab;
        p.c = width;
        p.cp = w;
        TRY(launch_pack<T>(c.embedding, p, embed.p, w, nullptr));
    }
    out_head = embed;
    if (c.head) {
        TRY(mat(&out_head, vocab, w));
        TRY(pack_rows(c.head, 1, vocab, vocab, vocab, 1, width, w, out_head.p, w));
    }
    norm_after = c.norm_after_sum != 0;
    if (norm_after) alpha = c.residual_scale;
    softcap = c.logit_softcap;
    TRY(vec(&final_norm, c.final_norm, 1, width, w));
    layers.resize(c.n_layers);
    for (int i = 0; i < c.n_layers; i++) TRY(load_layer(c.layers[i], layers[i]));

    // a convolution in the tail of a GEMV needs a lane per tap; norm staging rows in shared memory
    for (const MixLayer<T>& L : layers) {
        if (L.ch && !gemv_tail_fits<T>(w, L.taps)) fused_ok = false;
        for (const HeadPart& p : L.parts)
            if (p.taps && !gemv_tail_fits<T>(w, p.taps)) fused_ok = false;
        if (L.experts && !L.few) fused_ok = false;
    }
    if (!gemv_norm_fits<T>(w)) fused_ok = false;

    const bool loop = c.loop_times != 1 && c.loop_stop > c.loop_start;
    for (int i = 0; i < c.n_layers;) {
        if (loop && i == c.loop_start) {
            for (int p = 0; p < c.loop_times; p++)
                for (int j = c.loop_start; j < c.loop_stop; j++) order.emplace_back(j, c.loop_inject && p > 0 && j == c.loop_start);
            i = c.loop_stop;
        } else {
            order.emplace_back(i++, false);
        }
    }
    for (const auto& o : order) inject = inject || o.second;

    rows_cap = max_seq < kMaxRows ? max_seq : kMaxRows;
    if (rows_cap < max_batch) rows_cap = max_batch;
    const size_t R = rows_cap;
    const int ar = rows_cap < kAbsorbRows ? rows_cap : kAbsorbRows;
    size_t n_proj = 0, n_mixed = 0, n_ch = 0, n_x = 0, n_f32 = 0, n_q = 0, n_o = 0, n_ws = 0, n_k = 0, n_v = 0, n_rec = 0;
    auto up = [](size_t& a, size_t b) { if (b > a) a = b; };
    size_t n_heads_o = 0, n_scan = 0, n_z = 0, n_top = 0, n_gather = 0, n_hidden = 0, n_experts = 0;
    for (const MixLayer<T>& L : layers) {
        if (!L.experts) up(n_mixed, L.ff);
        up(n_mixed, L.out.ld);
        up(n_proj, L.parts.empty() ? L.in.rows : L.in_ld);
        for (const HeadPart& p : L.parts) {
            if (p.type == TLLM_MIXER_ATTENTION) {
                up(n_ws, grouped_workspace_floats(p.heads, p.vdim));
            } else {
                const bool delta = p.type == TLLM_MIXER_DELTA_RULE;
                up(n_heads_o, (size_t)p.heads * p.vdim);
                up(n_scan, matrix_scan_workspace(sizeof(T) == 2, delta, rows_cap, p.heads, p.kv_heads, p.dim, p.vdim));
                if (delta) up(n_ch, p.conv_channels());
            }
            up(n_f32, L.n_f32);
        }
        if (L.experts) {
            const size_t few = (size_t)(rows_cap < kFewRows ? rows_cap : kFewRows) * L.top, many = expert_rows(rows_cap, L.top, L.experts);
            up(n_z, L.router.rows);
            up(n_top, L.top);
            up(n_gather, many);
            up(n_hidden, (few > many ? few : many) * L.ff);
            up(n_experts, L.experts);
        }
        if (!L.parts.empty()) continue;
        if (L.type == TLLM_MIXER_LATENT_ATTENTION) {
            up(n_q, (size_t)L.heads * (L.rank + L.rot));
            up(n_o, (size_t)L.heads * L.rank);
            up(n_ws, latent_workspace_floats(ar, L.heads, L.rank));
            up(n_k, (size_t)L.heads * L.dim);
            up(n_v, (size_t)L.heads * L.vdim);
        } else {
            up(n_ch, L.ch);
            up(n_x, L.x.rows);
            up(n_f32, L.type == TLLM_MIXER_SELECTIVE_SCAN ? L.ch : 2 * L.ch);
            up(n_rec, scan_record_floats(1, rows_cap, L.ch, L.type == TLLM_MIXER_SELECTIVE_SCAN ? L.state : 1));
        }
    }
    auto some = [](size_t n) { return n ? n : (size_t)8; };
    TRY(dev_alloc(&x, R * w, true));
    TRY(dev_alloc(&x2, (size_t)kFewRows * w, true));
    if (inject) TRY(dev_alloc(&emb, R * w, true));
    TRY(dev_alloc(&y, R * w, true));
    TRY(dev_alloc(&h, R * w, true));
    TRY(dev_alloc(&proj, some(R * n_proj), true));
    TRY(dev_alloc(&mixed, some(R * n_mixed), true));
    TRY(dev_alloc(&conv_out, some(R * n_ch), true));
    TRY(dev_alloc(&xdbc, some(R * n_x), true));
    TRY(dev_alloc(&f32buf, some(R * n_f32), true));
    TRY(dev_alloc(&q_abs, some(ar * n_q), true));
    TRY(dev_alloc(&o_lat, some(ar * n_o), true));
    TRY(dev_alloc(&ws, some(n_ws), true));
    TRY(dev_alloc(&rec, some(n_rec), true));
    TRY(dev_alloc(&heads_o, some(R * n_heads_o), true));
    TRY(dev_alloc(&scan_ws, some(n_scan), true));
    TRY(dev_alloc(&router_z, some(R * n_z), true));
    TRY(dev_alloc(&part_w, some(R * n_top), true));
    TRY(dev_alloc(&chosen, some(R * n_top), true));
    TRY(dev_alloc(&part_row, some(R * n_top), true));
    TRY(dev_alloc(&gathered, some(n_gather * w), true));
    TRY(dev_alloc(&expert_out, some(n_gather * w), true));
    TRY(dev_alloc(&hidden, some(n_hidden), true));
    TRY(dev_alloc(&counts, some(2 * n_experts), true));
    TRY(dev_alloc(&group, some(3 * n_gather / kGroupRows), true));
    TRY(dev_alloc(&groups, 1, true));
    if (sizeof(T) == 2) {
        TRY(dev_alloc(&kx, some(max_seq * n_k), true));
        TRY(dev_alloc(&vx, some(max_seq * n_v), true));
    }
    TRY(dev_alloc(&logits, (size_t)max_batch * vocab, true));
    TRY(dev_alloc(&want_dev, R, true));
    for (const auto& o : order) {
        const MixLayer<T>& L = layers[o.first];
        RunState<T> rs;
        for (size_t i = 0; i < L.parts.size(); i++) TRY(part_state(L.parts[i], &rs.part[i]));
        if (!L.parts.empty()) {
            runs.push_back(rs);
            continue;
        }
        if (L.type == TLLM_MIXER_LATENT_ATTENTION) {
            rs.cache_slot = (size_t)max_seq * (L.rank + L.rot);
            TRY(dev_alloc(&rs.cache, rs.cache_slot * max_batch, true));
        } else {
            rs.conv_slot = (size_t)(L.taps - 1) * L.ch;
            rs.rec_slot = (size_t)L.ch * (L.type == TLLM_MIXER_SELECTIVE_SCAN ? L.state : 1);
            TRY(dev_alloc(&rs.conv, some(rs.conv_slot * max_batch), true));
            TRY(dev_alloc(&rs.rec, rs.rec_slot * max_batch, true));
            backup_bytes += rs.conv_slot * sizeof(T) + rs.rec_slot * sizeof(float);
        }
        runs.push_back(rs);
    }
    if (cudaDeviceSynchronize() != cudaSuccess) return fail(TLLM_ERR_LAUNCH, "mixed decoder: %s", cudaGetErrorString(cudaGetLastError()));
    return TLLM_OK;
}

// ---------------------------------------------------------------------------
// Sequences
// ---------------------------------------------------------------------------
template <typename T>
int MixedDecoder<T>::advance(int seq, int n_seq, int start_pos, int count)
{
    for (int b = seq; b < seq + n_seq; b++)
        if (start_pos > 0 && (recurrent ? start_pos != len[b] : start_pos > len[b]))
            return fail(TLLM_ERR_SHAPE, "decoder: position %d does not continue the sequence of slot %d (%d tokens so far)", start_pos, b, len[b]);
    for (int b = seq; b < seq + n_seq; b++) len[b] = start_pos + count;
    return TLLM_OK;
}

template <typename T>
int MixedDecoder<T>::copy_sequence(int seq, bool save, cudaStream_t s)
{
    if (!backup_bytes) return TLLM_OK;
    int st;
    if (!backup) TRY(dev_alloc(&backup, backup_bytes, false));
    uint8_t* p = backup;
    auto one = [&](void* state, size_t bytes) {
        if (bytes) cudaMemcpyAsync(save ? p : state, save ? state : p, bytes, cudaMemcpyDeviceToDevice, s);
        p += bytes;
    };
    for (RunState<T>& r : runs) {
        for (PartState<T>& p : r.part) {
            if (!p.rec) continue;
            one(p.rec + (size_t)seq * p.rec_slot, p.rec_slot * sizeof(float));
            one(p.conv + (size_t)seq * p.conv_slot, p.conv_slot * sizeof(T));
        }
        if (!r.rec) continue;
        one(r.rec + (size_t)seq * r.rec_slot, r.rec_slot * sizeof(float));
        one(r.conv + (size_t)seq * r.conv_slot, r.conv_slot * sizeof(T));
    }
    return check_launch("decoder: state copy");
}

// ---------------------------------------------------------------------------
// One step
// ---------------------------------------------------------------------------
template <>
bool MixedDecoder<float>::use_expanded(const LatentArgs<float>&) const { return false; }

template <>
int MixedDecoder<float>::expanded(const MixLayer<float>&, const RunState<float>&, const LatentArgs<float>&, cudaStream_t) { return TLLM_ERR_SHAPE; }

// Operations of the two forms (the expansion of the context runs as a GEMM, several times the
// rate of the attention kernels; softmax weights enter the second product twice).
template <>
bool MixedDecoder<bf16>::use_expanded(const LatentArgs<bf16>& a) const
{
    if (a.g.rows() <= kFewRows || !latent_expanded_supported(a)) return false;
    const double n = a.g.seq_len, ctx = a.g.start_pos + n;
    const double absorbed = n * ctx * (3.0 * a.rank + a.rot);
    const double expanded = ctx * 0.25 * a.rank * (a.dim + a.vdim) + n * ctx * (a.dim + a.rot + 2.0 * a.vdim);
    return expanded < absorbed;
}

template <>
int MixedDecoder<bf16>::expanded(const MixLayer<bf16>& L, const RunState<bf16>& R, const LatentArgs<bf16>& a, cudaStream_t s)
{
    int st;
    const int ctx = a.g.start_pos + a.g.seq_len, ldc = L.rank + L.rot;
    const bf16* cache = R.cache + (size_t)a.g.first_slot * R.cache_slot;
    TRY(project(L.k_up, cache, ldc, L.rank, kx, L.k_up.rows, false, ctx, s));
    TRY(project(L.v_up, cache, ldc, L.rank, vx, L.v_up.rows, false, ctx, s));
    return launch_latent_expanded(a, kx, vx, mixed, s);
}

template <typename T>
int MixedDecoder<T>::attention_inner(const MixLayer<T>& L, const RunState<T>& R, const StepGeo& g, cudaStream_t s)
{
    int st;
    const int rows = g.rows(), ldp = L.in.rows, H = L.heads, dq = L.dim + L.rot, dk = L.rank + L.rot;
    LatentArgs<T> a;
    a.proj = proj;
    a.ld = ldp;
    a.kv_off = H * dq;
    a.gate = L.head_gate ? proj + H * dq + dk : nullptr;
    a.gate_ld = ldp;
    a.heads = H;
    a.dim = L.dim;
    a.rot = L.rot;
    a.rot_true = L.rot_true;
    a.rot_dims = L.rot_dims;
    a.vdim = L.vdim;
    a.rank = L.rank;
    a.rank_true = L.rank_true;
    a.kv_norm = L.kv_norm;
    a.eps = eps;
    a.rope = L.rope;
    a.cache = R.cache;
    a.slot_stride = R.cache_slot;
    a.max_seq = max_seq;
    a.sink = L.sink;
    a.scale = L.scale;
    a.g = g;
    if (use_expanded(a)) {
        TRY(launch_latent_prep<T>(a, nullptr, s));
        TRY(expanded(L, R, a, s));
    } else {
        // row chunks of one sequence, or whole steps of several
        const int chunk = g.n_seq > 1 ? rows : kAbsorbRows;
        for (int r0 = 0; r0 < rows; r0 += chunk) {
            const int n = rows - r0 < chunk ? rows - r0 : chunk;
            LatentArgs<T> c = a;
            c.proj = proj + (size_t)r0 * ldp;
            if (a.gate) c.gate = a.gate + (size_t)r0 * ldp;
            if (g.n_seq == 1) {
                c.g.seq_len = n;
                c.g.start_pos = g.start_pos + r0;
            }
            TRY(launch_latent_prep<T>(c, q_abs, s));
            LinearArgs<T> l;
            l.w = L.k_up_t.p;
            l.ldw = L.k_up_t.ld;
            l.w_rows = L.rank;
            l.x = c.proj;
            l.ldx = ldp;
            l.x_batch = dq;
            l.y = q_abs;
            l.ldy = H * dk;
            l.y_batch = dk;
            l.M = n;
            l.N = L.rank;
            l.K = L.dim;
            l.batch = H;
            TRY(linear(l, s));
            TRY(launch_latent_absorbed<T>(c, q_abs, o_lat, ws, s));
            LinearArgs<T> v;
            v.w = L.v_up.p;
            v.ldw = L.v_up.ld;
            v.w_rows = L.vdim;
            v.x = o_lat;
            v.ldx = H * L.rank;
            v.x_batch = L.rank;
            v.y = mixed + (size_t)r0 * H * L.vdim;
            v.ldy = H * L.vdim;
            v.y_batch = L.vdim;
            v.M = n;
            v.N = L.vdim;
            v.K = L.rank;
            v.batch = H;
            v.gate = c.gate;
            v.gate_ld = ldp;
            TRY(linear(v, s));
        }
    }
    return TLLM_OK;
}

template <typename T>
ScanArgs<T> MixedDecoder<T>::scan_args(const MixLayer<T>& L, const RunState<T>& R, const StepGeo& g) const
{
    ScanArgs<T> a;
    a.x = conv_out;
    a.bc = xdbc;
    a.ld_bc = L.x.rows;
    a.b_off = L.dt8;
    a.c_off = L.dt8 + L.st8;
    if (scan_takes_dt(g.seq_len, L.state)) {
        a.dt_w = L.dt.p;
        a.dt_bias = L.dt_bias;
        a.dt_rank = L.dt8;
    } else {
        a.dt = f32buf;
    }
    a.z = proj + L.ch;
    a.ld_z = 2 * L.ch;
    a.a2 = L.a2;
    a.d = L.d;
    a.state = R.rec;
    a.slot_stride = R.rec_slot;
    a.y = mixed;
    a.channels = L.ch;
    a.states = L.state;
    a.rec = rec;
    a.g = g;
    return a;
}

template <typename T>
LinearArgs<T> MixedDecoder<T>::gates_args(const MixLayer<T>& L, int n_rows) const
{
    LinearArgs<T> l;
    l.w = L.gates.p;
    l.ldw = L.block;
    l.w_rows = 2 * L.block;
    l.x = conv_out;
    l.ldx = L.ch;
    l.x_batch = L.block;
    l.y = f32buf;
    l.ldy = 2 * L.ch;
    l.y_batch = 2 * L.block;
    l.y_f32 = true;
    l.M = n_rows;
    l.N = 2 * L.block;
    l.K = L.block;
    l.batch = L.blocks;
    l.bias = L.gate_bias;
    l.act = kActSigmoid;
    return l;
}

template <typename T>
LinearArgs<T> MixedDecoder<T>::in_product(const MixLayer<T>& L, int n_rows) const
{
    LinearArgs<T> l = product(L.in, h, w, w, proj, L.parts.empty() ? L.in.rows : L.in_ld, false, n_rows, L.in_bias, L.in_act);
    l.act_lo = L.act_lo;
    l.act_hi = L.act_hi;
    l.f32_from = L.f32_from;
    l.y2 = f32buf;
    l.ldy2 = L.n_f32;
    return l;
}

template <typename T>
GroupedArgs<T> MixedDecoder<T>::grouped_args(const MixLayer<T>& L, const HeadPart& p, const PartState<T>& S, const StepGeo& g) const
{
    GroupedArgs<T> a;
    a.proj = proj;
    a.ld = L.in_ld;
    a.q_off = p.q;
    a.k_off = p.k;
    a.v_off = p.v;
    a.heads = p.heads;
    a.kv_heads = p.kv_heads;
    a.dim = p.dim;
    a.vdim = p.vdim;
    a.dim_true = p.dim_true;
    a.q_norm = p.q_norm;
    a.k_norm = p.k_norm;
    a.eps = eps;
    a.rope = p.rope;
    a.rot_dims = p.rot_dims;
    a.kc = S.k;
    a.vc = S.v;
    a.k_slot = S.k_slot;
    a.v_slot = S.v_slot;
    a.cache_rows = S.cache_rows;
    a.max_seq = max_seq;
    a.chunk = p.chunk;
    a.scale = p.scale;
    a.out_scale = p.out_scale;
    a.out = mixed + p.out;
    a.ld_out = L.out.ld;
    a.g = g;
    return a;
}

template <typename T>
MatrixScanArgs<T> MixedDecoder<T>::matrix_args(const MixLayer<T>& L, const HeadPart& p, const PartState<T>& S, const StepGeo& g) const
{
    MatrixScanArgs<T> a;
    a.delta = p.type == TLLM_MIXER_DELTA_RULE;
    const T* x = proj + p.q;
    a.ld = L.in_ld;
    if (a.delta) {                             // behind the convolution
        x = conv_out;
        a.ld = p.conv_channels();
        a.a = f32buf + p.a;
        a.b = f32buf + p.b;
        a.ld_ab = L.n_f32;
        a.neg_a = p.neg_a;
        a.dt_bias = p.dt_bias;
        a.q_scale = 1.f / std::sqrt((float)p.dim_true);
    } else {
        a.decay = p.decay;
    }
    a.q = x;
    a.k = x + (p.k - p.q);
    a.v = x + (p.v - p.q);
    a.heads = p.heads;
    a.kv_heads = p.kv_heads;
    a.dim = p.dim;
    a.vdim = p.vdim;
    a.state = S.rec;
    a.slot_stride = S.rec_slot;
    a.o = heads_o;
    a.ws = scan_ws;
    a.g = g;
    return a;
}

template <typename T>
GatedNormArgs<T> MixedDecoder<T>::out_norm_args(const MixLayer<T>& L, const HeadPart& p, int n_rows) const
{
    const bool per_head = p.type == TLLM_MIXER_DELTA_RULE;
    GatedNormArgs<T> n;
    n.o = heads_o;
    n.w = p.norm;
    n.gate = proj + p.gate;
    n.ld_gate = L.in_ld;
    n.act = p.gate_act;
    n.eps = eps;
    n.out_scale = p.out_scale;
    n.out = mixed + p.out;
    n.ld_out = L.out.ld;
    n.rows = n_rows;
    n.groups = per_head ? p.heads : 1;
    n.n = per_head ? p.vdim : p.heads * p.vdim;
    n.n_true = per_head ? p.vdim_true : p.heads * p.vdim_true;
    return n;
}

// Mixers of heads: proj (and f32buf) -> mixed.  conv_done: conv_out is there already.
template <typename T>
int MixedDecoder<T>::heads_inner(const MixLayer<T>& L, const RunState<T>& R, const StepGeo& g, bool conv_done, cudaStream_t s)
{
    int st;
    if (g.seq_len == 1 && L.parts.size() == 2 && L.parts[0].type == TLLM_MIXER_ATTENTION && L.parts[1].type == TLLM_MIXER_LINEAR_ATTENTION)
        return launch_heads_step<T>(grouped_args(L, L.parts[0], R.part[0], g), matrix_args(L, L.parts[1], R.part[1], g),
                                    out_norm_args(L, L.parts[1], g.rows()), ws, s);
    for (size_t i = 0; i < L.parts.size(); i++) {
        const HeadPart& p = L.parts[i];
        const PartState<T>& S = R.part[i];
        if (p.type == TLLM_MIXER_ATTENTION) {
            TRY(launch_grouped_attention<T>(grouped_args(L, p, S, g), ws, s));
            continue;
        }
        if (p.type == TLLM_MIXER_DELTA_RULE && !conv_done) {
            ConvArgs<T> c;
            c.x = proj + p.q;
            c.ldx = L.in_ld;
            c.w = p.conv;
            c.state = S.conv;
            c.slot_stride = S.conv_slot;
            c.y = conv_out;
            c.channels = p.conv_channels();
            c.taps = p.taps;
            c.act = p.in_act;
            c.g = g;
            TRY(launch_causal_conv<T>(c, s));
        }
        const GatedNormArgs<T> n = out_norm_args(L, p, g.rows());
        TRY(launch_matrix_scan<T>(matrix_args(L, p, S, g), &n, s));
    }
    return TLLM_OK;
}

// h -> mixed, the input of the output projection
template <typename T>
int MixedDecoder<T>::mixer_inner(const MixLayer<T>& L, const RunState<T>& R, const StepGeo& g, cudaStream_t s)
{
    int st;
    const int rows = g.rows(), ch = L.ch;
    if (!L.parts.empty()) {
        TRY(linear(in_product(L, rows), s));
        return heads_inner(L, R, g, false, s);
    }
    if (L.type == TLLM_MIXER_LATENT_ATTENTION) {
        TRY(project(L.in, h, w, w, proj, L.in.rows, false, rows, s));
        return attention_inner(L, R, g, s);
    }
    const bool scan = L.type == TLLM_MIXER_SELECTIVE_SCAN;
    TRY(project(L.in, h, w, w, proj, 2 * ch, false, rows, s, L.in_bias));
    ConvArgs<T> c;
    c.x = scan ? proj : proj + ch;              // scan: [x | z]; recurrence: [y | x]
    c.ldx = 2 * ch;
    c.w = L.conv;
    c.bias = L.conv_bias;
    c.state = R.conv;
    c.slot_stride = R.conv_slot;
    c.y = conv_out;
    c.channels = ch;
    c.taps = L.taps;
    c.act = scan ? kActSilu : kActNone;
    c.g = g;
    TRY(launch_causal_conv<T>(c, s));
    if (scan) {
        TRY(project(L.x, conv_out, ch, ch, xdbc, L.x.rows, false, rows, s));
        const ScanArgs<T> a = scan_args(L, R, g);
        if (!a.dt_w) TRY(project(L.dt, xdbc, L.x.rows, L.dt8, f32buf, ch, true, rows, s, L.dt_bias, kActSoftplus));
        return launch_selective_scan<T>(a, s);
    }
    TRY(linear(gates_args(L, rows), s));
    GatedScanArgs<T> a;
    a.u = conv_out;
    a.gates = f32buf;
    a.soft_lam = L.soft_lam;
    a.c = L.decay;
    a.y = proj;
    a.ld_y = 2 * ch;
    a.act = L.gate_act;
    a.state = R.rec;
    a.slot_stride = R.rec_slot;
    a.out = mixed;
    a.channels = ch;
    a.block = L.block;
    a.rec = rec;
    a.g = g;
    return launch_gated_scan<T>(a, s);
}

// h -> y
template <typename T>
int MixedDecoder<T>::mixer(const MixLayer<T>& L, const RunState<T>& R, const StepGeo& g, cudaStream_t s)
{
    int st;
    TRY(mixer_inner(L, R, g, s));
    return project(L.out, mixed, L.out.ld, L.out.ld, y, w, true, g.rows(), s);
}

// Mixture of experts: h (or the residual chain staged in the router's product, which leaves h) -> y
// for few rows, expert_out with part_row and part_w for many
template <typename T>
int MixedDecoder<T>::experts(const MixLayer<T>& L, int n_rows, const GemvNorm* norm, cudaStream_t s)
{
    int st;
    const LinearArgs<T> r = product(L.router, h, w, w, router_z, L.router.rows, true, n_rows);
    if (norm) {
        GemvNorm f = *norm;
        f.h_out = h;
        TRY(launch_dense_gemv_fused<T>(r, f, GemvTail<T>(), s));
    } else {
        TRY(linear(r, s));
    }
    ExpertArgs<T> a;
    a.z = router_z;
    a.ld_z = L.router.rows;
    a.experts = L.experts;
    a.top = L.top;
    a.h = h;
    a.rows = n_rows;
    a.w = w;
    a.ff = L.ff;
    a.gate_up = L.gate_up.p;
    a.down = L.down.p;
    a.act = L.ff_act;
    a.hidden = hidden;
    a.y = y;
    if (!gathers(L, n_rows)) return launch_experts_few<T>(a, s);
    a.counts = counts;
    a.chosen = chosen;
    a.part_row = part_row;
    a.part_w = part_w;
    a.gathered = gathered;
    a.group = group;
    a.groups = groups;
    TRY(launch_experts_gather<T>(a, s));
    const int m = expert_rows(n_rows, L.top, L.experts);
    LinearArgs<T> l = product(L.gate_up, gathered, w, w, hidden, L.ff, false, m, nullptr, L.ff_act);
    l.w_rows = 2 * L.ff;
    l.N = L.ff;
    l.glu = true;
    l.group = group;
    l.groups = groups;
    l.entries = L.experts;
    TRY(linear(l, s));
    LinearArgs<T> d = product(L.down, hidden, L.ff, L.ff, expert_out, w, false, m);
    d.w_rows = d.N = w;
    d.group = group;
    d.groups = groups;
    d.entries = L.experts;
    return linear(d, s);
}

// h (or the residual chain staged in the first product) -> y
template <typename T>
int MixedDecoder<T>::feed_forward(const MixLayer<T>& L, int n_rows, const GemvNorm* norm, cudaStream_t s)
{
    int st;
    if (L.experts) return experts(L, n_rows, norm, s);
    LinearArgs<T> l;
    l.w = L.gate_up.p;
    l.ldw = w;
    l.w_rows = 2 * L.ff;
    l.x = h;
    l.ldx = w;
    l.y = mixed;
    l.ldy = L.ff;
    l.M = n_rows;
    l.N = L.ff;
    l.K = w;
    l.act = L.ff_act;
    l.glu = true;
    TRY(norm ? launch_dense_gemv_fused<T>(l, *norm, GemvTail<T>(), s) : linear(l, s));
    return project(L.down, mixed, L.ff, L.ff, y, w, true, n_rows, s);
}

// residual = table[token]; h = its norm for the first layer
template <typename T>
int MixedDecoder<T>::embed_rows(const int* tokens, int rows, cudaStream_t s)
{
    NormArgs<T> a;
    a.x = x;
    a.h = h;
    a.rows = rows;
    a.width = width;
    a.w = w;
    a.eps = eps;
    a.table = embed.p;
    a.tokens = tokens;
    a.emb = inject ? emb : nullptr;
    a.w_next = norm_after ? nullptr : layers[order[0].first].norm1;
    return launch_norm_chain<T>(a, s);
}

// One new token of each of a few sequences, logits of all of them: the residual chain is staged
// in the products behind it, the convolution step and the gated recurrence step are tails of
// the products in front of them.  Launches per layer without / with feed-forward: latent attention
// 7 / 9, scan 4 / 6, recurrence 3 / 5; a routed feed-forward is one more.
template <typename T>
int MixedDecoder<T>::decode_step(const int* tokens, const StepGeo& g, float* out, cudaStream_t s)
{
    int st;
    const int rows = g.rows();
    TRY(embed_rows(tokens, rows, s));
    float *cur = x, *next = x2;
    const float *post = nullptr, *sum = nullptr;
    auto chain = [&](const float* w_next, const float* extra) {
        GemvNorm f;
        f.y = y;
        f.alpha = alpha;
        f.w_post = post;
        f.w_sum = sum;
        f.x_in = cur;
        f.x_out = next;
        f.extra = extra;
        f.w_next = w_next;
        f.width = width;
        f.eps = eps;
        std::swap(cur, next);
        return f;
    };
    for (size_t r = 0; r < order.size(); r++) {
        const MixLayer<T>& L = layers[order[r].first];
        const RunState<T>& R = runs[r];
        const GemvNorm f = r == 0 ? GemvNorm() : chain(norm_after ? nullptr : L.norm1, order[r].second ? emb : nullptr);
        const LinearArgs<T> in = in_product(L, rows);
        GemvTail<T> t;
        for (size_t i = 0; i < L.parts.size(); i++) {
            const HeadPart& p = L.parts[i];
            if (p.type != TLLM_MIXER_DELTA_RULE) continue;
            t.kind = kTailConv;
            t.lo = p.q;
            t.hi = p.q + p.conv_channels();
            t.taps = p.taps;
            t.act = p.in_act;
            t.w = p.conv;
            t.carried = R.part[i].conv;
            t.slot_stride = R.part[i].conv_slot;
            t.first_slot = g.first_slot;
            t.start_pos = g.start_pos;
            t.pos_dev = g.pos_dev;
            t.out = conv_out;
            t.ld_out = p.conv_channels();
        }
        if (L.parts.empty() && L.type != TLLM_MIXER_LATENT_ATTENTION) {
            const bool scan = L.type == TLLM_MIXER_SELECTIVE_SCAN;
            t.kind = kTailConv;
            t.lo = scan ? 0 : L.ch;
            t.hi = t.lo + L.ch;
            t.taps = L.taps;
            t.act = scan ? kActSilu : kActNone;
            t.w = L.conv;
            t.bias = L.conv_bias;
            t.carried = R.conv;
            t.slot_stride = R.conv_slot;
            t.first_slot = g.first_slot;
            t.start_pos = g.start_pos;
            t.pos_dev = g.pos_dev;
            t.out = conv_out;
            t.ld_out = L.ch;
        }
        TRY(launch_dense_gemv_fused<T>(in, f, t, s));
        if (!L.parts.empty()) {
            TRY(heads_inner(L, R, g, t.kind == kTailConv, s));
        } else if (L.type == TLLM_MIXER_LATENT_ATTENTION) {
            TRY(attention_inner(L, R, g, s));
        } else if (L.type == TLLM_MIXER_SELECTIVE_SCAN) {
            TRY(project(L.x, conv_out, L.ch, L.ch, xdbc, L.x.rows, false, rows, s));
            const ScanArgs<T> a = scan_args(L, R, g);
            if (!a.dt_w) TRY(project(L.dt, xdbc, L.x.rows, L.dt8, f32buf, L.ch, true, rows, s, L.dt_bias, kActSoftplus));
            TRY(launch_selective_scan<T>(a, s));
        } else {
            LinearArgs<T> l = gates_args(L, rows);
            l.N = L.block;
            t.kind = kTailGate;
            t.act = L.gate_act;
            t.soft_lam = L.soft_lam;
            t.decay = L.decay;
            t.y = proj;
            t.ld_y = 2 * L.ch;
            t.state = R.rec;
            t.slot_stride = R.rec_slot;
            t.out = mixed;
            TRY(launch_dense_gemv_fused<T>(l, GemvNorm(), t, s));
        }
        TRY(project(L.out, mixed, L.out.ld, L.out.ld, y, w, true, rows, s));
        post = L.norm1b;
        sum = norm_after ? L.norm1 : nullptr;
        if (L.has_ff()) {
            const GemvNorm n2 = chain(norm_after ? nullptr : L.norm2, nullptr);
            TRY(feed_forward(L, rows, &n2, s));
            post = L.norm2b;
            sum = norm_after ? L.norm2 : nullptr;
        }
    }
    return launch_dense_gemv_fused<T>(head_product(rows, out), chain(final_norm, nullptr), GemvTail<T>(), s);
}

template <typename T>
int MixedDecoder<T>::layers_pass(const int* tokens, const StepGeo& g, float* taps, size_t tap_stride, cudaStream_t s)
{
    int st;
    const int rows = g.rows();
    NormArgs<T> base;
    base.x = x;
    base.h = h;
    base.rows = rows;
    base.width = width;
    base.w = w;
    base.eps = eps;
    TRY(embed_rows(tokens, rows, s));
    base.y = y;
    base.alpha = alpha;
    for (size_t r = 0; r < order.size(); r++) {
        const MixLayer<T>& L = layers[order[r].first];
        TRY(mixer(L, runs[r], g, s));
        NormArgs<T> a = base;
        a.w_post = L.norm1b;
        a.w_sum = norm_after ? L.norm1 : nullptr;
        if (L.has_ff()) {
            a.w_next = norm_after ? nullptr : L.norm2;
            TRY(launch_norm_chain<T>(a, s));
            TRY(feed_forward(L, rows, nullptr, s));
            a = base;
            a.w_post = L.norm2b;
            a.w_sum = norm_after ? L.norm2 : nullptr;
            if (gathers(L, rows)) {
                a.y = nullptr;
                a.parts = expert_out;
                a.part_row = part_row;
                a.part_w = part_w;
                a.top = L.top;
            }
        }
        a.tap = taps ? taps + r * tap_stride : nullptr;
        a.tap_width = width;
        if (r + 1 < order.size()) {
            a.extra = order[r + 1].second ? emb : nullptr;
            a.w_next = norm_after ? nullptr : layers[order[r + 1].first].norm1;
        } else {
            a.h = nullptr;
        }
        TRY(launch_norm_chain<T>(a, s));
    }
    return TLLM_OK;
}

template <typename T>
LinearArgs<T> MixedDecoder<T>::head_product(int n, float* out) const
{
    LinearArgs<T> l = product(out_head, h, w, w, out, vocab, true, n, nullptr, softcap > 0.f ? kActSoftcap : kActNone);
    l.act_param = softcap;
    return l;
}

// final norm and output head of n rows of the residual stream
template <typename T>
int MixedDecoder<T>::head(const float* rows_x, const int* row_map, int n, float* out, cudaStream_t s)
{
    int st;
    NormArgs<T> a;
    a.x = const_cast<float*>(rows_x);
    a.row_map = row_map;
    a.w_next = final_norm;
    a.h = h;
    a.rows = n;
    a.width = width;
    a.w = w;
    a.eps = eps;
    TRY(launch_norm_chain<T>(a, s));
    return linear(head_product(n, out), s);
}

template <typename T>
int MixedDecoder<T>::forward(const int* tokens, int n, int start_pos, const int* pos_dev, int seq, int batch, cudaStream_t s)
{
    int st;
    if (batch > 0) {
        StepGeo g;
        g.n_seq = batch;
        g.start_pos = start_pos;
        if (fuses(g)) return decode_step(tokens, g, logits, s);
        TRY(layers_pass(tokens, g, nullptr, 0, s));
        return head(x, nullptr, batch, logits, s);
    }
    int last = 0;
    for (int t0 = 0; t0 < n; t0 += rows_cap) {
        StepGeo g;
        g.seq_len = n - t0 < rows_cap ? n - t0 : rows_cap;
        g.first_slot = seq;
        g.start_pos = start_pos + t0;
        g.pos_dev = pos_dev;
        if (n == 1 && fuses(g)) return decode_step(tokens, g, logits + (size_t)seq * vocab, s);
        TRY(layers_pass(tokens + t0, g, nullptr, 0, s));
        last = g.seq_len - 1;
    }
    return head(x + (size_t)last * w, nullptr, 1, logits + (size_t)seq * vocab, s);
}

template <typename T>
int MixedDecoder<T>::forward_logits(const int* tokens, int n, int start_pos, int seq, const int* want, int n_want, float* out, float* taps,
                                    cudaStream_t s)
{
    int st;
    for (int t0 = 0; t0 < n; t0 += rows_cap) {
        StepGeo g;
        g.seq_len = n - t0 < rows_cap ? n - t0 : rows_cap;
        g.first_slot = seq;
        g.start_pos = start_pos + t0;
        if (n == 1 && !taps && fuses(g)) {                       // the step that generation runs
            TRY(decode_step(tokens, g, logits + (size_t)seq * vocab, s));
            for (int i = 0; i < n_want; i++)
                cudaMemcpyAsync(out + (size_t)i * vocab, logits + (size_t)seq * vocab, (size_t)vocab * sizeof(float), cudaMemcpyDeviceToDevice, s);
            return check_launch("decoder_forward_logits");
        }
        TRY(layers_pass(tokens + t0, g, taps ? taps + (size_t)t0 * width : nullptr, (size_t)n * width, s));
        // runs of wanted tokens that lie in this portion
        for (int i = 0; i < n_want;) {
            std::vector<int> rows;
            int j = i;
            while (j < n_want && want[j] >= t0 && want[j] < t0 + g.seq_len && (int)rows.size() < rows_cap) rows.push_back(want[j++] - t0);
            if (rows.empty()) {
                i++;
                continue;
            }
            if (cudaMemcpyAsync(want_dev, rows.data(), rows.size() * sizeof(int), cudaMemcpyHostToDevice, s) != cudaSuccess ||
                cudaStreamSynchronize(s) != cudaSuccess)
                return fail(TLLM_ERR_LAUNCH, "decoder_forward_logits: %s", cudaGetErrorString(cudaGetLastError()));
            TRY(head(x, want_dev, (int)rows.size(), out + (size_t)i * vocab, s));
            i = j;
        }
    }
    return TLLM_OK;
}

#undef TRY

template <typename T>
int create_mixed(const tllm_b200_mixed_desc& c, int flags, int max_batch, void** out)
{
    MixedDecoder<T>* D = new MixedDecoder<T>();
    const int st = D->create(c, flags, max_batch);
    if (st) {
        delete D;
        return st;
    }
    *out = static_cast<Decoder*>(D);
    return TLLM_OK;
}

}  // namespace

}  // namespace tllm

using namespace tllm;

extern "C" {

int tllm_b200_mixed_decoder_create(const tllm_b200_mixed_desc* desc, int flags, int max_batch, void** out)
{
    if (!desc || !out || !desc->layers || !desc->embedding || !desc->final_norm) return fail(TLLM_ERR_NULL, "mixed_decoder_create: null argument");
    if (max_batch < 1 || max_batch > TLLM_DECODER_MAX_BATCH)
        return fail(TLLM_ERR_BATCH, "mixed_decoder_create: max_batch=%d outside 1..%d", max_batch, TLLM_DECODER_MAX_BATCH);
    const tllm_b200_mixed_desc& c = *desc;
    if (c.vocab_size < 1 || c.width < 1 || c.n_layers < 1 || c.max_seq_len < 1 || c.loop_start < 0 || c.loop_stop > c.n_layers || c.loop_times < 1)
        return fail(TLLM_ERR_SHAPE, "mixed_decoder_create: vocab=%d width=%d layers=%d max_seq_len=%d loop=%d..%d x %d", c.vocab_size, c.width,
                    c.n_layers, c.max_seq_len, c.loop_start, c.loop_stop, c.loop_times);
    const int st = check_device();
    if (st) return st;
    return (flags & TLLM_DECODER_FLOAT32) ? create_mixed<float>(c, flags, max_batch, out) : create_mixed<bf16>(c, flags, max_batch, out);
}

int tllm_b200_mixed_decoder_runs(void* decoder)
{
    return decoder ? static_cast<Decoder*>(decoder)->n_runs() : 0;
}

}  // extern "C"
