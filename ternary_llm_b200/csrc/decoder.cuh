// Base of the library's decoders: one loaded model together with the state of the sequences
// it serves.  A model class supplies the pass over its layers; the handle, the greedy decode
// loop and the C entry points (decoder.cu) are shared.
#pragma once
#include <vector>

#include "common.cuh"

namespace tllm {

struct Decoder {
    int flags = 0, max_batch = 1;  // sequences (slots) with their own cache and state
    int max_seq = 0, vocab = 0;
    bool logits_f32 = false;       // FP16 otherwise
    // device-side state of the graph-replayed decode loop
    int* state = nullptr;          // [0] token, [1] position, [2] step
    int* history = nullptr;        // generated tokens
    int history_cap = 0;
    float* am_val = nullptr;
    int* am_idx = nullptr;
    unsigned* am_counter = nullptr;
    cudaStream_t stream = nullptr; // owned, for generate()
    cudaGraphExec_t step_graph = nullptr;
    std::vector<void*> owned;

    virtual ~Decoder();
    // One pass of the layer stack.
    //   batch == 0: n tokens of sequence `seq` at positions start_pos.. (pos_dev != nullptr: one
    //               token whose position is read from device memory, start_pos ignored);
    //   batch  > 0: one token of each of the sequences 0..batch-1 (n == batch), all at position
    //               start_pos; logits for every sequence.
    virtual int forward(const int* tokens, int n, int start_pos, const int* pos_dev, int seq, int batch, cudaStream_t s) = 0;
    virtual int reset(cudaStream_t s) = 0;
    virtual void* logits_row(int seq) = 0;
    // Called before `count` tokens of each of n_seq sequences are run from start_pos on: a model
    // with recurrent state refuses positions that do not continue the sequence.
    virtual int advance(int seq, int n_seq, int start_pos, int count)
    {
        (void)seq, (void)n_seq, (void)start_pos, (void)count;
        return TLLM_OK;
    }
    // Copy of what a repeated step would not rewrite (recurrent state).
    virtual int save_sequence(int seq, cudaStream_t s) { (void)seq, (void)s; return TLLM_OK; }
    virtual int restore_sequence(int seq, cudaStream_t s) { (void)seq, (void)s; return TLLM_OK; }
    // Logits of n_want of the n tokens (places among them, ascending or not), FP32 [n_want, vocab];
    // taps: when not null, the residual stream after every layer run.
    virtual int forward_logits(const int* tokens, int n, int start_pos, int seq, const int* want_host, int n_want, float* out, float* taps,
                               cudaStream_t s)
    {
        (void)tokens, (void)n, (void)start_pos, (void)seq, (void)want_host, (void)n_want, (void)out, (void)taps, (void)s;
        return fail(TLLM_ERR_SHAPE, "decoder_forward_logits: this model returns the logits of the last token only");
    }

    virtual int n_runs() const { return 0; }       // layer runs of a pass, where forward_logits exists

    int init_common(int flags, int max_batch, int max_seq, int vocab);
    int dev_alloc_bytes(void** out, size_t bytes, bool zero);
    template <typename T>
    int dev_alloc(T** out, size_t n, bool zero)
    {
        void* p = nullptr;
        const int st = dev_alloc_bytes(&p, n * sizeof(T), zero);
        *out = static_cast<T*>(p);
        return st;
    }
};

}  // namespace tllm
