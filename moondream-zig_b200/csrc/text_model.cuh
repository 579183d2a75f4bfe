// The text models' host-side objects, shared by model.cu (the request, the step and the generation loop of every text
// model, and the Phi-style decoder's layers) and stack.cu (the layers of the layer-stack decoders).
#pragma once

#include "md_internal.cuh"

#include "../../include/moondream_b200_model.h"

struct DevPtr {
    void* p = nullptr;
    size_t cap = 0;
    DevPtr() = default;
    DevPtr(const DevPtr&) = delete;
    DevPtr& operator=(const DevPtr&) = delete;
    ~DevPtr() { if (p) cudaFree(p); }
    int ensure(md_ctx* ctx, size_t bytes) {
        if (cap >= bytes) return MD_OK;
        if (ctx->capturing) return md_fail(ctx, MD_ERR_UNSUPPORTED, "buffer growth during graph capture");
        if (p) {
            MD_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
            MD_CUDA(ctx, cudaFree(p));
            p = nullptr;
            cap = 0;
        }
        MD_CUDA(ctx, cudaMalloc(&p, bytes));
        cap = bytes;
        return MD_OK;
    }
    template <class T> T* as() const { return reinterpret_cast<T*>(p); }
};

struct md_stack;          // the layers of a layer-stack decoder (stack.cu)
struct md_stack_request;  // what a request of one holds between and during steps

struct md_text_model {
    md_ctx* ctx = nullptr;
    md_text_weights w = {};   // layer-stack models: the sizes only
    std::vector<const uint16_t*> ln_w, ln_b, wqkv, bqkv, wout, bout, wfc1, bfc1, wfc2, bfc2;
    md_stack* stack = nullptr;
};

struct md_text_request {
    md_text_model* model = nullptr;
    std::vector<__half*> kc, vc;  // per layer [n_heads][max_seq][head_dim]
    md_stack_request* stack = nullptr;
    size_t pos = 0;               // host mirror of *pos_dev
    int* pos_dev = nullptr;       // [0] tokens held, [1] current copy of the convolution states (layer-stack models)
    // activations of one forward over `rows` rows
    DevPtr hidden, ln, qkv, attn, attn_out, fc1, logits, ln_last;
    DevPtr mlp_part;  // up to four f32 [8, dim] partial products of fc2 (the decode layer whose MLP runs as two half-width chains)
    // device-side generation state
    DevPtr cur_token, sampled, tokens_out, forced, step, logits_all, pos_ptrs;
    md_graph* graph = nullptr;
    uint64_t graph_gen = 0, prefill_graph_gen = 0;  // md_ctx::generation the graphs were captured under
    size_t graph_steps = 0;
    bool graph_forced = false, graph_logits = false;
    // a prefill of the same shape at the same position seen twice is captured and replayed
    md_graph* prefill_graph = nullptr;
    size_t prefill_S = 0, prefill_pos = 0, seen_S = 0, seen_pos = ~(size_t)0;
};

// While alive, the kernels that implement the programmatic-dependent-launch protocol (GEMV, tcgen05 GEMM and
// attention, LayerNorm, rope) are launched dependent on their predecessor: each starts its set-up while the
// previous one drains and waits (griddepcontrol.wait) before touching global memory.
struct PdlScope {
    md_ctx* c;
    int old;
    explicit PdlScope(md_ctx* cc) : c(cc), old(cc->pdl) { c->pdl = 1; }
    ~PdlScope() { c->pdl = old; }
};

// The second stream of a layer that runs as two chains of kernels, and its events (model.cu).
int md_side_stream(md_ctx* ctx);

// ---- stack.cu ----------------------------------------------------------------------------------------------
int md_stack_destroy(md_stack* s);
int md_stack_request_create(md_text_request* req);
void md_stack_request_destroy(md_text_request* req);
int md_stack_request_reset(md_text_request* req);
// Make room for steps of `rows` rows in the request's activation buffers (before any capture).
int md_stack_reserve(md_text_request* req, size_t rows);
// The layers over `rows` rows of each of `seqs` requests, from token ids in device memory ([seqs * rows], in
// reqs[0]'s buffers); decode: one row per request at the position in device memory, else one request at pos0.
int md_stack_layers(md_text_model* m, md_text_request* const* reqs, size_t seqs, size_t rows,
                    const unsigned long long* tokens_dev, bool decode, size_t pos0);
// Final norm and head over `n` of the `step_rows` rows md_stack_layers has run: rows_dev (device indices), or the first n.
// logits f32 [n, vocab].  sampled != null (n <= 8, zero before the call): the rows' greedy samples, as keys for
// advance_kernel if the call returns with *keys set, as indices otherwise.
int md_stack_head(md_text_model* m, md_text_request* r0, size_t step_rows, const int* rows_dev, size_t n, float* logits,
                  unsigned long long* sampled, bool* keys);
int md_stack_copy_stream(md_text_request* req, size_t layer, float* out, size_t rows);
