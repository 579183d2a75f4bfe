// Layer-stack decoders: the layers of a text model that is described layer by layer (md_stack_weights).  Requests, the
// step entry point, the generation loop, its graphs and the batched form are those of every text model (model.cu); here
// is what a request keeps per layer (key caches, recurrent states, convolution tails) and the kernels of one pass.
#include "stack.cuh"
#include "text_model.cuh"

#include <algorithm>

struct md_stack {
    md_stack_weights w = {};
    std::vector<md_stack_layer> layers;
    size_t elem = 2;                 // bytes of T
    size_t max_in = 0, max_o = 0, max_ff = 0, max_ssq = 0, max_top = 0, max_experts = 0, max_moe_ff = 0;
    size_t kv_bytes = 0;             // key caches of one request
    size_t state_floats = 0;         // recurrent states and convolution tails of one request
    std::vector<size_t> kv_off, rec_off, conv1_off, conv2_off;   // per layer; bytes / floats
};

struct md_stack_request {
    DevPtr keys;      // all key caches
    DevPtr state;     // all f32 states, zeroed by a reset
    DevPtr x[2], h, in, o, y, ff, ssq;
    DevPtr route, score, sel, rank, slot, count, tile_expert, n_blocks, xs, act, ys;
    DevPtr trace;     // [layers][rows][width] when stack_trace is set
    size_t cap_rows = 0, trace_rows = 0;
};

namespace {

md_glue base_glue(const md_stack& s, size_t rows, size_t seqs) {
    md_glue g;
    g.width = (int)s.w.width;
    g.rows = (int)rows;
    g.seqs = (int)seqs;
    g.eps = s.w.eps;
    g.mult = s.w.residual_mult;
    g.taps = (int)s.w.taps;
    return g;
}

size_t align_up(size_t v, size_t a) { return (v + a - 1) / a * a; }

// Where the output of a product that ends a sublayer lies when a step has T rows in all: f32 rows for a few tokens, T rows
// otherwise.
bool rows_f32(const md_stack& s, size_t T) { return T <= 8 || s.w.dtype == MD_DTYPE_F32; }

// The residual update that follows layer `i`'s mixer (ff == false) or feed-forward, for steps of seqs x rows tokens.
// A function of the shapes alone, so that a replayed step leaves the same thing behind as an issued one.
md_glue update_after(const md_stack& s, md_stack_request* b, size_t i, bool ff, size_t rows, size_t seqs) {
    const md_stack_layer& l = s.layers[i];
    md_glue g = base_glue(s, rows, seqs);
    g.w_post = ff ? l.norm2b : l.norm1b;
    if (ff && l.ff == MD_FF_MOE && md_moe_sorted(s.w.dtype, s.w.width, rows * seqs)) {
        g.slot = b->slot.as<int>(), g.score = b->score.as<float>(), g.top = (int)l.top;
        g.y = b->ys.p;
        return g;
    }
    if (rows_f32(s, rows * seqs)) g.y_f32 = b->y.as<float>();
    else g.y = b->y.p;
    if (!ff && l.mixer == MD_MIXER_LIGHTNING) {
        g.ssq = b->ssq.as<float>();
        g.ssq_parts = md_lightning_ssq_parts((int)l.heads, (int)l.vdim);
        g.ssq_n = (int)(l.heads * l.vdim);
    }
    return g;
}

// Which of the two residual buffers holds the stream after all layers (every residual update goes to the other one).
int final_x(const md_stack& s) {
    int n = 0;
    for (const md_stack_layer& l : s.layers) n += l.ff == MD_FF_NONE ? 1 : 2;
    return n & 1;
}

}  // namespace

extern "C" int md_stack_model_create(md_ctx* ctx, const md_stack_weights* w, md_text_model** out) {
    if (!ctx) return MD_ERR_INVALID_ARG;
    if (!w || !out || !w->layers || !w->embed || !w->head || !w->final_norm)
        return md_fail(ctx, MD_ERR_INVALID_ARG, "md_stack_model_create: null argument");
    if (w->dtype != MD_DTYPE_BF16 && w->dtype != MD_DTYPE_F32)
        return md_fail(ctx, MD_ERR_UNSUPPORTED, "layer-stack models run in bfloat16 or float32");
    if (!w->n_layers || !w->width || !w->vocab || !w->max_seq || w->taps < 1 || w->taps > MD_STACK_MAX_TAPS)
        return md_fail(ctx, MD_ERR_INVALID_ARG, "md_stack_model_create: sizes (1 <= taps <= %d)", MD_STACK_MAX_TAPS);
    md_stack s;
    s.w = *w;
    s.elem = w->dtype == MD_DTYPE_F32 ? 4 : 2;
    s.layers.assign(w->layers, w->layers + w->n_layers);
    s.w.layers = nullptr;
    for (size_t i = 0; i < s.layers.size(); ++i) {
        const md_stack_layer& l = s.layers[i];
        const bool attn = l.mixer == MD_MIXER_WINDOW_ATTENTION;
        if (!attn && l.mixer != MD_MIXER_LIGHTNING) return md_fail(ctx, MD_ERR_UNSUPPORTED, "layer %zu: unknown mixer %d", i, l.mixer);
        if (!l.heads || !l.dim || !l.w_in || !l.w_out || !l.norm1 || !l.norm1b || !l.conv1)
            return md_fail(ctx, MD_ERR_INVALID_ARG, "layer %zu: missing mixer weights or sizes", i);
        if (attn && (!l.kv_heads || l.heads % l.kv_heads || l.vdim != l.dim || !l.r1 || !l.r2))
            return md_fail(ctx, MD_ERR_INVALID_ARG, "layer %zu: attention needs kv_heads dividing heads, vdim == dim, r1 and r2", i);
        if (!attn && (!l.vdim || !l.decay || !l.mix_norm))
            return md_fail(ctx, MD_ERR_INVALID_ARG, "layer %zu: lightning needs vdim, decay and its norm", i);
        const size_t used = attn ? (l.heads + l.kv_heads) * l.dim + l.heads : 2 * l.heads * (l.dim + l.vdim);
        if (l.in_rows != align_up(used, 8))
            return md_fail(ctx, MD_ERR_SHAPE, "layer %zu: w_in has %zu rows, expected %zu", i, l.in_rows, align_up(used, 8));
        if (l.ff != MD_FF_NONE) {
            if (!l.norm2 || !l.norm2b || !l.conv2 || !l.w_gate_up || !l.w_down || (l.act != MD_ACT_GELU_TANH && l.act != MD_ACT_SILU))
                return md_fail(ctx, MD_ERR_INVALID_ARG, "layer %zu: missing feed-forward weights", i);
            if (l.ff_pad != align_up(l.ff_dim, MD_GLU_BLOCK)) return md_fail(ctx, MD_ERR_SHAPE, "layer %zu: ff_pad", i);
        }
        if (l.ff == MD_FF_MOE && (!l.router || !l.experts || !l.top || l.top > l.experts))
            return md_fail(ctx, MD_ERR_INVALID_ARG, "layer %zu: router", i);
        s.kv_off.push_back(s.kv_bytes);
        if (attn) s.kv_bytes += align_up(l.kv_heads * w->max_seq * l.dim * s.elem, 256);
        s.rec_off.push_back(s.state_floats);
        if (!attn) s.state_floats += align_up(l.heads * l.dim * l.vdim, 64);
        s.conv1_off.push_back(s.state_floats);
        s.state_floats += align_up(2 * (w->taps - 1) * w->width, 64);
        s.conv2_off.push_back(s.state_floats);
        if (l.ff != MD_FF_NONE) s.state_floats += align_up(2 * (w->taps - 1) * w->width, 64);
        s.max_in = std::max(s.max_in, l.in_rows);
        s.max_o = std::max(s.max_o, l.heads * l.vdim);
        if (!attn) s.max_ssq = std::max(s.max_ssq, (size_t)md_lightning_ssq_parts((int)l.heads, (int)l.vdim));
        if (l.ff == MD_FF_DENSE) s.max_ff = std::max(s.max_ff, l.ff_pad);
        if (l.ff == MD_FF_MOE) {
            s.max_top = std::max(s.max_top, l.top);
            s.max_experts = std::max(s.max_experts, l.experts);
            s.max_moe_ff = std::max(s.max_moe_ff, l.ff_pad);
        }
    }
    md_text_model* m = new md_text_model();
    m->ctx = ctx;
    m->w.n_layers = w->n_layers;
    m->w.dim = w->width;
    m->w.vocab = w->vocab;
    m->w.max_seq = w->max_seq;
    m->stack = new md_stack(s);
    *out = m;
    return MD_OK;
}

int md_stack_destroy(md_stack* s) {
    delete s;
    return MD_OK;
}

int md_stack_request_create(md_text_request* req) {
    md_ctx* ctx = req->model->ctx;
    const md_stack& s = *req->model->stack;
    md_stack_request* r = req->stack = new md_stack_request();
    MD_TRY(r->keys.ensure(ctx, std::max<size_t>(s.kv_bytes, 256)));
    MD_TRY(r->state.ensure(ctx, std::max<size_t>(s.state_floats, 64) * sizeof(float)));
    if (s.max_experts) {
        const size_t bytes = md_moe_route_floats(s.max_experts) * sizeof(float);
        MD_TRY(r->route.ensure(ctx, bytes));
        MD_CUDA(ctx, cudaMemsetAsync(r->route.p, 0, bytes, ctx->stream));
    }
    MD_TRY(md_stack_reserve(req, MD_STACK_MAX_SEQS));
    return md_stack_request_reset(req);
}

void md_stack_request_destroy(md_text_request* req) {
    delete req->stack;
    req->stack = nullptr;
}

// A key is only read after the same request wrote it, so the caches need no clearing; the recurrences start from zero.
int md_stack_request_reset(md_text_request* req) {
    md_ctx* ctx = req->model->ctx;
    MD_CUDA(ctx, cudaMemsetAsync(req->stack->state.p, 0, req->stack->state.cap, ctx->stream));
    return MD_OK;
}

int md_stack_reserve(md_text_request* req, size_t rows) {
    md_ctx* ctx = req->model->ctx;
    const md_stack& s = *req->model->stack;
    md_stack_request* r = req->stack;
    const bool trace = ctx->stack_trace != 0;
    if (trace && r->trace_rows < rows) {
        MD_TRY(r->trace.ensure(ctx, s.layers.size() * rows * s.w.width * sizeof(float)));
        r->trace_rows = rows;
    }
    if (r->cap_rows >= rows) return MD_OK;
    // the buffers are about to move: captured steps that point at them are stale
    if (req->graph) { md_graph_destroy(ctx, req->graph); req->graph = nullptr; }
    if (req->prefill_graph) { md_graph_destroy(ctx, req->prefill_graph); req->prefill_graph = nullptr; }
    const size_t W = s.w.width, E = s.elem;
    for (auto& x : r->x) MD_TRY(x.ensure(ctx, rows * W * sizeof(float)));
    MD_TRY(r->h.ensure(ctx, rows * W * E));
    MD_TRY(r->in.ensure(ctx, rows * s.max_in * E));
    MD_TRY(r->o.ensure(ctx, rows * s.max_o * E));
    MD_TRY(r->y.ensure(ctx, rows * W * sizeof(float)));
    if (s.max_ff) MD_TRY(r->ff.ensure(ctx, rows * s.max_ff * E));
    if (s.max_ssq) MD_TRY(r->ssq.ensure(ctx, rows * s.max_ssq * sizeof(float)));
    if (s.max_experts) {
        MD_TRY(r->score.ensure(ctx, rows * s.max_top * sizeof(float)));
        MD_TRY(r->sel.ensure(ctx, rows * s.max_top * sizeof(int)));
        MD_TRY(r->rank.ensure(ctx, rows * s.max_top * sizeof(int)));
        MD_TRY(r->slot.ensure(ctx, rows * s.max_top * sizeof(int)));
        MD_TRY(r->count.ensure(ctx, s.max_experts * sizeof(int)));
        size_t cap = 0;
        for (const md_stack_layer& l : s.layers)
            if (l.ff == MD_FF_MOE) cap = std::max(cap, md_moe_sorted_rows(rows, (int)l.experts, (int)l.top));
        MD_TRY(r->tile_expert.ensure(ctx, cap / MD_GROUP_ROWS * sizeof(int)));
        MD_TRY(r->n_blocks.ensure(ctx, sizeof(int)));
        MD_TRY(r->xs.ensure(ctx, cap * W * E));
        MD_TRY(r->act.ensure(ctx, cap * s.max_moe_ff * E));
        MD_TRY(r->ys.ensure(ctx, cap * W * E));
    }
    r->cap_rows = rows;
    return MD_OK;
}

int md_stack_layers(md_text_model* m, md_text_request* const* reqs, size_t seqs, size_t rows,
                    const unsigned long long* tokens_dev, bool decode, size_t pos0) {
    md_ctx* ctx = m->ctx;
    const md_stack& s = *m->stack;
    md_stack_request* b = reqs[0]->stack;   // the activations of the step
    const size_t W = s.w.width, T = seqs * rows;
    const int dt = s.w.dtype;
    int cur = 0;
    md_glue next = base_glue(s, rows, seqs);   // the residual update the next kernel has to make
    next.tokens = tokens_dev;
    next.embed = s.w.embed;
    next.vocab = (int)s.w.vocab;
    auto run_glue = [&](md_glue g, const float* w_pre, const float* conv, const std::vector<size_t>& off, size_t layer) -> int {
        g.x = g.tokens ? nullptr : b->x[cur].as<float>();
        g.x_out = b->x[cur ^ 1].as<float>();
        cur ^= 1;
        g.w_pre = w_pre;
        g.conv = conv;
        for (size_t i = 0; i < seqs; ++i) {
            g.state[i] = reqs[i]->stack->state.as<float>() + off[layer];
            g.state_slot[i] = reqs[i]->pos_dev + 1;
        }
        g.out = b->h.p;
        return md_launch_glue(ctx, dt, g);
    };
    auto trace = [&](size_t layer) -> int {   // x holds the stream after `layer`
        if (ctx->stack_trace && !ctx->capturing && b->trace.p)
            MD_CUDA(ctx, cudaMemcpyAsync(b->trace.as<float>() + layer * b->trace_rows * W, b->x[cur].p, T * W * sizeof(float),
                                         cudaMemcpyDeviceToDevice, ctx->stream));
        return MD_OK;
    };
    auto out_product = [&](const void* a, const void* w, size_t K) -> int {   // ends a sublayer
        md_lin ep;
        if (rows_f32(s, T)) ep.out_f32 = b->y.as<float>();
        return md_linear(ctx, dt, a, w, b->y.p, T, W, K, ep);
    };
    for (size_t i = 0; i < s.layers.size(); ++i) {
        const md_stack_layer& l = s.layers[i];
        MD_TRY(run_glue(next, l.norm1, l.conv1, s.conv1_off, i));
        if (i > 0) MD_TRY(trace(i - 1));
        md_lin in;
        in.bias = l.b_in;
        if (l.mixer == MD_MIXER_LIGHTNING) in.silu_cols = in.sigmoid_from = (int)(l.heads * (2 * l.dim + l.vdim));
        else in.sigmoid_from = (int)((l.heads + l.kv_heads) * l.dim);
        MD_TRY(md_linear(ctx, dt, b->h.p, l.w_in, b->in.p, T, l.in_rows, W, in));
        if (l.mixer == MD_MIXER_WINDOW_ATTENTION) {
            md_win_attn a;
            a.heads = (int)l.heads, a.kv_heads = (int)l.kv_heads, a.dim = (int)l.dim;
            a.scale = l.scale, a.window = (int)l.window, a.keep_first = (int)l.keep_first;
            a.r1 = l.r1, a.r2 = l.r2;
            a.qkg = b->in.p, a.row_stride = (int)l.in_rows, a.out = b->o.p;
            a.rows = (int)rows, a.seqs = (int)seqs, a.max_seq = s.w.max_seq, a.pos0 = (int)pos0;
            for (size_t q = 0; q < seqs; ++q) {
                a.kc[q] = reqs[q]->stack->keys.as<char>() + s.kv_off[i];
                a.pos_dev[q] = decode ? reqs[q]->pos_dev : nullptr;
            }
            MD_TRY(md_launch_window_attention(ctx, dt, a, decode));
        } else {
            md_lightning a;
            a.heads = (int)l.heads, a.dim = (int)l.dim, a.vdim = (int)l.vdim;
            a.decay = l.decay, a.norm_w = l.mix_norm;
            a.qkvg = b->in.p, a.row_stride = (int)l.in_rows, a.out = b->o.p;
            a.ssq = b->ssq.as<float>();
            a.ssq_parts = md_lightning_ssq_parts(a.heads, a.vdim);
            a.rows = (int)rows, a.seqs = (int)seqs;
            for (size_t q = 0; q < seqs; ++q) a.state[q] = reqs[q]->stack->state.as<float>() + s.rec_off[i];
            MD_TRY(md_launch_lightning(ctx, dt, a, decode));
        }
        MD_TRY(out_product(b->o.p, l.w_out, l.heads * l.vdim));
        next = update_after(s, b, i, false, rows, seqs);
        if (l.ff == MD_FF_NONE) continue;
        MD_TRY(run_glue(next, l.norm2, l.conv2, s.conv2_off, i));
        if (l.ff == MD_FF_DENSE) {
            md_lin up;
            up.glu = l.act;
            MD_TRY(md_linear(ctx, dt, b->h.p, l.w_gate_up, b->ff.p, T, 2 * l.ff_pad, W, up));
            MD_TRY(out_product(b->ff.p, l.w_down, l.ff_pad));
        } else {
            md_moe e;
            e.width = (int)W, e.experts = (int)l.experts, e.top = (int)l.top, e.ff = (int)l.ff_dim, e.ff_pad = (int)l.ff_pad;
            e.act = l.act, e.router = l.router, e.w_gu = l.w_gate_up, e.w_down = l.w_down;
            md_moe_buffers mb;
            mb.score = b->score.as<float>(), mb.sel = b->sel.as<int>(), mb.rank = b->rank.as<int>(), mb.slot = b->slot.as<int>();
            mb.count = b->count.as<int>(), mb.tile_expert = b->tile_expert.as<int>(), mb.n_blocks = b->n_blocks.as<int>();
            mb.xs = b->xs.p, mb.act = b->act.p, mb.ys = b->ys.p, mb.y_f32 = b->y.as<float>(), mb.route = b->route.as<float>();
            MD_TRY(md_launch_moe(ctx, dt, e, b->h.p, T, mb));
        }
        next = update_after(s, b, i, true, rows, seqs);
    }
    if (ctx->stack_trace && !ctx->capturing) {
        md_glue g = next;
        g.x = b->x[cur].as<float>();
        g.x_out = b->x[cur ^ 1].as<float>();
        g.w_pre = s.w.final_norm;
        g.out = b->h.p;
        MD_TRY(md_launch_glue(ctx, dt, g));
        cur ^= 1;
        MD_TRY(trace(s.layers.size() - 1));
    }
    return MD_OK;
}

int md_stack_head(md_text_model* m, md_text_request* r0, size_t step_rows, const int* rows_dev, size_t n, float* logits,
                  unsigned long long* sampled, bool* keys) {
    md_ctx* ctx = m->ctx;
    const md_stack& s = *m->stack;
    md_stack_request* b = r0->stack;
    const size_t last = s.layers.size() - 1;
    md_glue g = update_after(s, b, last, s.layers[last].ff != MD_FF_NONE, step_rows, 1);
    g.x = b->x[final_x(s)].as<float>();
    g.x_out = nullptr;
    g.w_pre = s.w.final_norm;
    g.conv = nullptr;
    g.out = b->h.p;
    if (rows_dev) {
        g.gather = rows_dev;
        g.rows = (int)n;
        g.seqs = 1;
    } else {
        g.rows = 1;
        g.seqs = (int)n;
    }
    MD_TRY(md_launch_glue(ctx, s.w.dtype, g));
    md_lin head;
    head.out_f32 = logits;
    const bool fused = sampled && s.w.dtype == MD_DTYPE_BF16 && n <= 8 && md_gemv_lin_supported(b->h.p, s.w.head, s.w.width);
    if (fused) head.amax = sampled;
    MD_TRY(md_linear(ctx, s.w.dtype, b->h.p, s.w.head, nullptr, n, s.w.vocab, s.w.width, head));
    if (sampled && !fused) MD_TRY(md_launch_argmax_f32(ctx, logits, s.w.vocab, s.w.vocab, n, sampled));
    if (keys) *keys = fused;
    return MD_OK;
}

int md_stack_copy_stream(md_text_request* req, size_t layer, float* out, size_t rows) {
    md_ctx* ctx = req->model->ctx;
    const md_stack& s = *req->model->stack;
    md_stack_request* b = req->stack;
    if (layer >= s.layers.size() || !out || !b->trace.p || rows > b->trace_rows)
        return md_fail(ctx, MD_ERR_INVALID_ARG, "md_text_layer_stream: nothing recorded for layer %zu (set stack_trace)", layer);
    MD_CUDA(ctx, cudaMemcpyAsync(out, b->trace.as<float>() + layer * b->trace_rows * s.w.width, rows * s.w.width * sizeof(float),
                                 cudaMemcpyDeviceToHost, ctx->stream));
    return md_check_flags(ctx);
}
