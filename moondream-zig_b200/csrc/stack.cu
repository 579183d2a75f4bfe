// Layer-stack decoders: the layers of a text model that is described layer by layer (md_stack_weights).  Requests, the
// step entry point, the generation loop, its graphs and the batched form are those of every text model (model.cu); here
// is what a request keeps per layer (key caches, recurrent states, convolution tails) and the kernels of one pass.
#include "stack.cuh"
#include "text_model.cuh"

#include <algorithm>
#include <memory>

struct md_stack {
    md_stack_weights w = {};
    std::vector<md_stack_layer> layers;
    size_t elem = 2;                 // bytes of T
    bool parallel = false;           // MD_LAYER_PARALLEL
    size_t max_in = 0, max_o = 0, max_ff = 0, max_ssq = 0, max_top = 0, max_choices = 0, max_experts = 0, max_moe_ff = 0, max_shared = 0;
    size_t max_cq = 0, max_q = 0, max_qa = 0;   // latent attention, per row
    size_t kv_bytes = 0;             // key caches of one request
    size_t state_floats = 0;         // recurrent states and convolution tails of one request
    std::vector<size_t> kv_off, rec_off, conv1_off, conv2_off;   // per layer; bytes / floats
    struct Rotation { size_t dims; float base; DevPtr table; };   // one table per pair of dimensions and base
    std::vector<std::unique_ptr<Rotation>> rotations;
    std::vector<const float*> rope;  // per layer
    // keys and values a prompt's portion expands, one buffer for all layers and requests (steps follow one another)
    DevPtr kv;
};

struct md_stack_request {
    DevPtr keys;      // all key caches
    DevPtr state;     // all f32 states, zeroed by a reset
    DevPtr x[2], h, in, o, y, ff, ssq;
    DevPtr h2, y2;              // parallel layers: the feed-forward's input and output
    DevPtr cq, q, qa;           // latent attention
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
        g.slot = b->slot.as<int>(), g.score = b->score.as<float>(), g.top = (int)(l.top + (l.shared_ff ? 1 : 0));
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

// The same for a parallel layer's two sublayers.
md_parallel_glue update_after_parallel(const md_stack& s, md_stack_request* b, size_t i, size_t rows, size_t seqs) {
    const md_stack_layer& l = s.layers[i];
    md_parallel_glue g;
    g.width = (int)s.w.width;
    g.rows = (int)(rows * seqs);
    g.eps = s.w.eps;
    const bool f32 = rows_f32(s, rows * seqs);
    if (f32) g.b[0].y_f32 = b->y.as<float>();
    else g.b[0].y = b->y.p;
    g.b[0].scale = l.ls1;
    if (l.ff == MD_FF_NONE) return g;
    g.b[1].scale = l.ls2;
    if (l.ff == MD_FF_MOE && md_moe_sorted(s.w.dtype, s.w.width, rows * seqs)) {
        g.b[1].slot = b->slot.as<int>(), g.b[1].score = b->score.as<float>(), g.b[1].top = (int)(l.top + (l.shared_ff ? 1 : 0));
        g.b[1].y = b->ys.p;
    } else if (f32) {
        g.b[1].y_f32 = b->y2.as<float>();
    } else {
        g.b[1].y = b->y2.p;
    }
    return g;
}

// Which of the two residual buffers holds the stream after all layers (every residual update goes to the other one; parallel
// layers update in place).
int final_x(const md_stack& s) {
    if (s.parallel) return 0;
    int n = 0;
    for (const md_stack_layer& l : s.layers) n += l.ff == MD_FF_NONE ? 1 : 2;
    return n & 1;
}

}  // namespace

static int add_rotation(md_ctx* ctx, md_stack& s, size_t dims, float base) {
    for (const auto& r : s.rotations)
        if (r->dims == dims && r->base == base) {
            s.rope.push_back(r->table.as<float>());
            return MD_OK;
        }
    auto r = std::make_unique<md_stack::Rotation>();
    r->dims = dims, r->base = base;
    MD_TRY(r->table.ensure(ctx, std::max<size_t>(s.w.max_seq * dims * sizeof(float), 256)));
    MD_TRY(md_launch_rotation_table(ctx, r->table.as<float>(), s.w.max_seq, dims, base));
    s.rope.push_back(r->table.as<float>());
    s.rotations.push_back(std::move(r));
    return MD_OK;
}

extern "C" int md_stack_model_create(md_ctx* ctx, const md_stack_weights* w, md_text_model** out) {
    if (!ctx) return MD_ERR_INVALID_ARG;
    if (!w || !out || !w->layers || !w->embed || !w->head || !w->final_norm)
        return md_fail(ctx, MD_ERR_INVALID_ARG, "md_stack_model_create: null argument");
    if (w->dtype != MD_DTYPE_BF16 && w->dtype != MD_DTYPE_F32)
        return md_fail(ctx, MD_ERR_UNSUPPORTED, "layer-stack models run in bfloat16 or float32");
    if (!w->n_layers || !w->width || !w->vocab || !w->max_seq || w->taps < 1 || w->taps > MD_STACK_MAX_TAPS)
        return md_fail(ctx, MD_ERR_INVALID_ARG, "md_stack_model_create: sizes (1 <= taps <= %d)", MD_STACK_MAX_TAPS);
    auto own = std::make_unique<md_stack>();
    md_stack& s = *own;
    s.w = *w;
    s.elem = w->dtype == MD_DTYPE_F32 ? 4 : 2;
    s.layers.assign(w->layers, w->layers + w->n_layers);
    s.w.layers = nullptr;
    s.parallel = s.layers[0].form == MD_LAYER_PARALLEL;
    for (size_t i = 0; i < s.layers.size(); ++i) {
        const md_stack_layer& l = s.layers[i];
        const bool attn = l.mixer == MD_MIXER_WINDOW_ATTENTION, latent = l.mixer == MD_MIXER_LATENT_ATTENTION;
        const bool lightning = l.mixer == MD_MIXER_LIGHTNING;
        if (!attn && !latent && !lightning) return md_fail(ctx, MD_ERR_UNSUPPORTED, "layer %zu: unknown mixer %d", i, l.mixer);
        if ((l.form != MD_LAYER_SANDWICH && l.form != MD_LAYER_PARALLEL) || (l.form == MD_LAYER_PARALLEL) != s.parallel)
            return md_fail(ctx, MD_ERR_UNSUPPORTED, "layer %zu: form %d (all layers have the same form)", i, l.form);
        if (!l.heads || !l.dim || !l.w_in || !l.w_out || !l.norm1)
            return md_fail(ctx, MD_ERR_INVALID_ARG, "layer %zu: missing mixer weights or sizes", i);
        if (!s.parallel && (!l.norm1b || !l.conv1)) return md_fail(ctx, MD_ERR_INVALID_ARG, "layer %zu: norm1b and conv1", i);
        if (s.parallel && (l.conv1 || l.conv2 || l.norm1b || l.norm2b))
            return md_fail(ctx, MD_ERR_INVALID_ARG, "layer %zu: a parallel layer has no convolution and no norm1b or norm2b", i);
        if (s.parallel && lightning) return md_fail(ctx, MD_ERR_UNSUPPORTED, "layer %zu: lightning attention in a parallel layer", i);
        if (attn && (!l.kv_heads || l.heads % l.kv_heads || l.vdim != l.dim || !l.r1 || !l.r2))
            return md_fail(ctx, MD_ERR_INVALID_ARG, "layer %zu: attention needs kv_heads dividing heads, vdim == dim, r1 and r2", i);
        if (latent && (!l.vdim || !l.q_rank || !l.kv_rank || (l.rot_dim % 2) || !l.q_norm || !l.kv_norm || !l.sink || !l.w_uq || !l.w_ukv ||
                       !(l.rope_base > 0.f)))
            return md_fail(ctx, MD_ERR_INVALID_ARG, "layer %zu: latent attention's sizes, norms, sink or matrices", i);
        if (lightning && (!l.vdim || !l.decay || !l.mix_norm))
            return md_fail(ctx, MD_ERR_INVALID_ARG, "layer %zu: lightning needs vdim, decay and its norm", i);
        const size_t used = attn ? (l.heads + l.kv_heads) * l.dim + l.heads : latent ? l.q_rank + l.kv_rank + l.rot_dim
                                 : 2 * l.heads * (l.dim + l.vdim);
        if (l.in_rows != align_up(used, 8))
            return md_fail(ctx, MD_ERR_SHAPE, "layer %zu: w_in has %zu rows, expected %zu", i, l.in_rows, align_up(used, 8));
        if (l.ff != MD_FF_NONE) {
            if (!l.norm2 || (!s.parallel && (!l.norm2b || !l.conv2)) || !l.w_gate_up || !l.w_down || l.act < MD_ACT_GELU_TANH ||
                l.act > MD_ACT_CLAMPED)
                return md_fail(ctx, MD_ERR_INVALID_ARG, "layer %zu: missing feed-forward weights", i);
            if (l.ff_pad != align_up(l.ff_dim, MD_GLU_BLOCK)) return md_fail(ctx, MD_ERR_SHAPE, "layer %zu: ff_pad", i);
        }
        if (l.ff == MD_FF_MOE && (!l.router || !l.experts || !l.top || l.top > l.experts))
            return md_fail(ctx, MD_ERR_INVALID_ARG, "layer %zu: router", i);
        if (l.ff == MD_FF_MOE && l.router_kind != MD_ROUTER_LOGISTIC && l.router_kind != MD_ROUTER_SOFTMAX)
            return md_fail(ctx, MD_ERR_UNSUPPORTED, "layer %zu: unknown router %d", i, l.router_kind);
        if (l.shared_ff && (l.ff != MD_FF_MOE || !l.shared_gate_up || !l.shared_down || l.shared_pad != align_up(l.shared_ff, MD_GLU_BLOCK)))
            return md_fail(ctx, MD_ERR_INVALID_ARG, "layer %zu: shared expert", i);
        s.kv_off.push_back(s.kv_bytes);
        if (latent) {
            s.kv_bytes += align_up(w->max_seq * l.kv_rank * s.elem, 256) + align_up(w->max_seq * l.rot_dim * s.elem, 256);
            s.max_cq = std::max(s.max_cq, l.q_rank);
            s.max_q = std::max(s.max_q, l.heads * (l.dim + l.rot_dim));
            s.max_qa = std::max(s.max_qa, l.heads * (l.kv_rank + l.rot_dim));
            MD_TRY(add_rotation(ctx, s, l.rot_dim, l.rope_base));
        } else {
            s.rope.push_back(nullptr);
        }
        if (attn) s.kv_bytes += align_up(l.kv_heads * w->max_seq * l.dim * s.elem, 256);
        s.rec_off.push_back(s.state_floats);
        if (lightning) s.state_floats += align_up(l.heads * l.dim * l.vdim, 64);
        s.conv1_off.push_back(s.state_floats);
        s.state_floats += align_up(2 * (w->taps - 1) * w->width, 64);
        s.conv2_off.push_back(s.state_floats);
        if (l.ff != MD_FF_NONE) s.state_floats += align_up(2 * (w->taps - 1) * w->width, 64);
        s.max_in = std::max(s.max_in, l.in_rows);
        s.max_o = std::max(s.max_o, l.heads * l.vdim);
        if (lightning) s.max_ssq = std::max(s.max_ssq, (size_t)md_lightning_ssq_parts((int)l.heads, (int)l.vdim));
        if (l.ff == MD_FF_DENSE) s.max_ff = std::max(s.max_ff, l.ff_pad);
        if (l.ff == MD_FF_MOE) {
            s.max_top = std::max(s.max_top, l.top);
            s.max_choices = std::max(s.max_choices, l.top + (l.shared_ff ? 1 : 0));
            if (l.shared_ff) s.max_shared = std::max(s.max_shared, l.shared_pad);
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
    m->stack = own.release();
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
    if (s.max_ff || s.max_shared) MD_TRY(r->ff.ensure(ctx, rows * std::max(s.max_ff, s.max_shared) * E));
    if (s.parallel) {
        MD_TRY(r->h2.ensure(ctx, rows * W * E));
        MD_TRY(r->y2.ensure(ctx, rows * W * sizeof(float)));
    }
    if (s.max_cq) {
        MD_TRY(r->cq.ensure(ctx, rows * s.max_cq * E));
        MD_TRY(r->q.ensure(ctx, rows * s.max_q * E));
        MD_TRY(r->qa.ensure(ctx, MD_STACK_MAX_SEQS * s.max_qa * E));
    }
    if (s.max_ssq) MD_TRY(r->ssq.ensure(ctx, rows * s.max_ssq * sizeof(float)));
    if (s.max_experts) {
        MD_TRY(r->score.ensure(ctx, rows * s.max_choices * sizeof(float)));
        MD_TRY(r->sel.ensure(ctx, rows * s.max_top * sizeof(int)));
        MD_TRY(r->rank.ensure(ctx, rows * s.max_top * sizeof(int)));
        MD_TRY(r->slot.ensure(ctx, rows * s.max_choices * sizeof(int)));
        MD_TRY(r->count.ensure(ctx, s.max_experts * sizeof(int)));
        size_t cap = 0;
        for (const md_stack_layer& l : s.layers)
            if (l.ff == MD_FF_MOE) cap = std::max(cap, md_moe_sorted_rows(rows, (int)l.experts, (int)l.top));
        MD_TRY(r->tile_expert.ensure(ctx, cap / MD_GROUP_ROWS * sizeof(int)));
        MD_TRY(r->n_blocks.ensure(ctx, sizeof(int)));
        MD_TRY(r->xs.ensure(ctx, cap * W * E));
        MD_TRY(r->act.ensure(ctx, (cap * s.max_moe_ff + MD_STACK_MAX_SEQS * s.max_shared) * E));
        MD_TRY(r->ys.ensure(ctx, (cap + (s.max_shared ? rows : 0)) * W * E));
    }
    r->cap_rows = rows;
    return MD_OK;
}

namespace {

// What one pass over the layers works with.
struct Pass {
    md_ctx* ctx;
    md_stack& s;
    md_text_request* const* reqs;
    size_t seqs, rows, T;     // rows per sequence, rows in all
    bool decode;
    size_t pos0;
    md_stack_request* b;      // the activations of the step
};

int out_product(const Pass& p, const void* a, const void* w, DevPtr& y, size_t K) {   // ends a sublayer
    md_lin ep;
    if (rows_f32(p.s, p.T)) ep.out_f32 = y.as<float>();
    return md_linear(p.ctx, p.s.w.dtype, a, w, y.p, p.T, p.s.w.width, K, ep);
}

int window_mixer(const Pass& p, size_t i) {
    const md_stack_layer& l = p.s.layers[i];
    md_win_attn a;
    a.heads = (int)l.heads, a.kv_heads = (int)l.kv_heads, a.dim = (int)l.dim;
    a.scale = l.scale, a.window = (int)l.window, a.keep_first = (int)l.keep_first;
    a.r1 = l.r1, a.r2 = l.r2;
    a.qkg = p.b->in.p, a.row_stride = (int)l.in_rows, a.out = p.b->o.p;
    a.rows = (int)p.rows, a.seqs = (int)p.seqs, a.max_seq = p.s.w.max_seq, a.pos0 = (int)p.pos0;
    for (size_t q = 0; q < p.seqs; ++q) {
        a.kc[q] = p.reqs[q]->stack->keys.as<char>() + p.s.kv_off[i];
        a.pos_dev[q] = p.decode ? p.reqs[q]->pos_dev : nullptr;
    }
    return md_launch_window_attention(p.ctx, p.s.w.dtype, a, p.decode);
}

int lightning_mixer(const Pass& p, size_t i) {
    const md_stack_layer& l = p.s.layers[i];
    md_lightning a;
    a.heads = (int)l.heads, a.dim = (int)l.dim, a.vdim = (int)l.vdim;
    a.decay = l.decay, a.norm_w = l.mix_norm;
    a.qkvg = p.b->in.p, a.row_stride = (int)l.in_rows, a.out = p.b->o.p;
    a.ssq = p.b->ssq.as<float>();
    a.ssq_parts = md_lightning_ssq_parts(a.heads, a.vdim);
    a.rows = (int)p.rows, a.seqs = (int)p.seqs;
    for (size_t q = 0; q < p.seqs; ++q) a.state[q] = p.reqs[q]->stack->state.as<float>() + p.s.rec_off[i];
    return md_launch_lightning(p.ctx, p.s.w.dtype, a, p.decode);
}

int latent_mixer(const Pass& p, size_t i) {
    const md_stack_layer& l = p.s.layers[i];
    md_stack_request* b = p.b;
    md_latent a;
    a.heads = (int)l.heads, a.dim = (int)l.dim, a.rot = (int)l.rot_dim, a.vdim = (int)l.vdim;
    a.q_rank = (int)l.q_rank, a.kv_rank = (int)l.kv_rank;
    a.scale = l.scale, a.eps = p.s.w.eps, a.window = (int)l.window;
    a.q_norm = l.q_norm, a.kv_norm = l.kv_norm, a.sink = l.sink, a.rope = p.s.rope[i];
    a.w_uq = l.w_uq, a.w_ukv = l.w_ukv, a.w_ukt = l.w_ukt;
    a.in = b->in.p, a.row_stride = (int)l.in_rows;
    a.cq = b->cq.p, a.q = b->q.p, a.qa = b->qa.p, a.out = b->o.p;
    a.rows = (int)p.rows, a.seqs = (int)p.seqs, a.max_seq = p.s.w.max_seq, a.pos0 = (int)p.pos0;
    for (size_t q = 0; q < p.seqs; ++q) {
        char* at = p.reqs[q]->stack->keys.as<char>() + p.s.kv_off[i];
        a.cc[q] = at;
        a.kr[q] = at + align_up(p.s.w.max_seq * l.kv_rank * p.s.elem, 256);
        a.pos_dev[q] = p.decode ? p.reqs[q]->pos_dev : nullptr;
    }
    if (!p.decode && md_latent_expands(p.s.w.dtype, a)) {
        const size_t bytes = md_latent_keys(p.rows, l.window, p.s.w.max_seq) * l.heads * (l.dim + l.vdim) * p.s.elem;
        if (p.s.kv.cap < bytes) {
            MD_TRY(p.s.kv.ensure(p.ctx, bytes));
            p.ctx->generation++;       // recorded passes of any request point at the old buffer
        }
        a.kv = p.s.kv.p;
    }
    return md_launch_latent_attention(p.ctx, p.s.w.dtype, a, p.decode);
}

// b->h -> b->y
int run_mixer(const Pass& p, size_t i) {
    const md_stack_layer& l = p.s.layers[i];
    md_lin in;
    in.bias = l.b_in;
    if (l.mixer == MD_MIXER_LIGHTNING) in.silu_cols = in.sigmoid_from = (int)(l.heads * (2 * l.dim + l.vdim));
    else if (l.mixer == MD_MIXER_WINDOW_ATTENTION) in.sigmoid_from = (int)((l.heads + l.kv_heads) * l.dim);
    MD_TRY(md_linear(p.ctx, p.s.w.dtype, p.b->h.p, l.w_in, p.b->in.p, p.T, l.in_rows, p.s.w.width, in));
    if (l.mixer == MD_MIXER_WINDOW_ATTENTION) MD_TRY(window_mixer(p, i));
    else if (l.mixer == MD_MIXER_LIGHTNING) MD_TRY(lightning_mixer(p, i));
    else MD_TRY(latent_mixer(p, i));
    return out_product(p, p.b->o.p, l.w_out, p.b->y, l.heads * l.vdim);
}

// h -> y (or the sorted rows)
int run_ff(const Pass& p, size_t i, const void* h, DevPtr& y) {
    const md_stack_layer& l = p.s.layers[i];
    md_stack_request* b = p.b;
    if (l.ff == MD_FF_DENSE) {
        md_lin up;
        up.glu = l.act, up.glu_limit = l.act_limit, up.glu_alpha = l.act_alpha;
        MD_TRY(md_linear(p.ctx, p.s.w.dtype, h, l.w_gate_up, b->ff.p, p.T, 2 * l.ff_pad, p.s.w.width, up));
        return out_product(p, b->ff.p, l.w_down, y, l.ff_pad);
    }
    md_moe e;
    e.width = (int)p.s.w.width, e.experts = (int)l.experts, e.top = (int)l.top, e.ff_pad = (int)l.ff_pad;
    e.act = l.act, e.limit = l.act_limit, e.alpha = l.act_alpha;
    e.router_kind = l.router_kind, e.router = l.router, e.w_gu = l.w_gate_up, e.w_down = l.w_down;
    if (l.shared_ff) {
        e.shared_pad = (int)l.shared_pad, e.shared_limit = l.shared_limit;
        e.shared_gu = l.shared_gate_up, e.shared_down = l.shared_down;
    }
    md_moe_buffers mb;
    mb.score = b->score.as<float>(), mb.sel = b->sel.as<int>(), mb.rank = b->rank.as<int>(), mb.slot = b->slot.as<int>();
    mb.count = b->count.as<int>(), mb.tile_expert = b->tile_expert.as<int>(), mb.n_blocks = b->n_blocks.as<int>();
    mb.xs = b->xs.p, mb.act = b->act.p, mb.ys = b->ys.p, mb.y_f32 = y.as<float>(), mb.route = b->route.as<float>();
    mb.shared_act = b->ff.p;
    return md_launch_moe(p.ctx, p.s.w.dtype, e, h, p.T, mb);
}

int keep_stream(const Pass& p, size_t layer, int cur) {   // x[cur] holds the stream after `layer`
    const size_t W = p.s.w.width;
    if (p.ctx->stack_trace && !p.ctx->capturing && p.b->trace.p)
        MD_CUDA(p.ctx, cudaMemcpyAsync(p.b->trace.as<float>() + layer * p.b->trace_rows * W, p.b->x[cur].p, p.T * W * sizeof(float),
                                       cudaMemcpyDeviceToDevice, p.ctx->stream));
    return MD_OK;
}

int sandwich_layers(const Pass& p, const unsigned long long* tokens_dev) {
    md_ctx* ctx = p.ctx;
    const md_stack& s = p.s;
    md_stack_request* b = p.b;
    int cur = 0;
    md_glue next = base_glue(s, p.rows, p.seqs);   // the residual update the next kernel has to make
    next.tokens = tokens_dev;
    next.embed = s.w.embed;
    next.vocab = (int)s.w.vocab;
    auto run_glue = [&](md_glue g, const float* w_pre, const float* conv, const std::vector<size_t>& off, size_t layer) -> int {
        g.x = g.tokens ? nullptr : b->x[cur].as<float>();
        g.x_out = b->x[cur ^ 1].as<float>();
        cur ^= 1;
        g.w_pre = w_pre;
        g.conv = conv;
        for (size_t i = 0; i < p.seqs; ++i) {
            g.state[i] = p.reqs[i]->stack->state.as<float>() + off[layer];
            g.state_slot[i] = p.reqs[i]->pos_dev + 1;
        }
        g.out = b->h.p;
        return md_launch_glue(ctx, s.w.dtype, g);
    };
    for (size_t i = 0; i < s.layers.size(); ++i) {
        const md_stack_layer& l = s.layers[i];
        MD_TRY(run_glue(next, l.norm1, l.conv1, s.conv1_off, i));
        if (i > 0) MD_TRY(keep_stream(p, i - 1, cur));
        MD_TRY(run_mixer(p, i));
        next = update_after(s, b, i, false, p.rows, p.seqs);
        if (l.ff == MD_FF_NONE) continue;
        MD_TRY(run_glue(next, l.norm2, l.conv2, s.conv2_off, i));
        MD_TRY(run_ff(p, i, b->h.p, b->y));
        next = update_after(s, b, i, true, p.rows, p.seqs);
    }
    if (ctx->stack_trace && !ctx->capturing) {
        md_glue g = next;
        g.x = b->x[cur].as<float>();
        g.x_out = b->x[cur ^ 1].as<float>();
        g.w_pre = s.w.final_norm;
        g.out = b->h.p;
        MD_TRY(md_launch_glue(ctx, s.w.dtype, g));
        MD_TRY(keep_stream(p, s.layers.size() - 1, cur ^ 1));
    }
    return MD_OK;
}

// Both sublayers of a layer read the same row, so they run as two chains of kernels (the feed-forward's on the context's
// side stream) that meet in the next residual update.
int parallel_layers(const Pass& p, const unsigned long long* tokens_dev) {
    md_ctx* ctx = p.ctx;
    const md_stack& s = p.s;
    md_stack_request* b = p.b;
    MD_TRY(md_side_stream(ctx));
    cudaStream_t main_stream = ctx->stream;
    md_parallel_glue next;
    next.width = (int)s.w.width, next.rows = (int)p.T, next.eps = s.w.eps;
    next.tokens = tokens_dev, next.embed = s.w.embed, next.vocab = (int)s.w.vocab;
    for (size_t i = 0; i < s.layers.size(); ++i) {
        const md_stack_layer& l = s.layers[i];
        next.x = next.tokens ? nullptr : b->x[0].as<float>();
        next.x_out = b->x[0].as<float>();
        next.w[0] = l.norm1, next.out[0] = b->h.p;
        next.w[1] = l.norm2, next.out[1] = l.ff == MD_FF_NONE ? nullptr : b->h2.p;
        MD_TRY(md_launch_parallel_glue(ctx, s.w.dtype, next));
        if (i > 0) MD_TRY(keep_stream(p, i - 1, 0));
        if (l.ff != MD_FF_NONE) {
            MD_CUDA(ctx, cudaEventRecord(ctx->ev_fork, main_stream));
            MD_CUDA(ctx, cudaStreamWaitEvent(ctx->side_stream, ctx->ev_fork, 0));
            ctx->stream = ctx->side_stream;
            int st = run_ff(p, i, b->h2.p, b->y2);
            if (st == MD_OK && cudaEventRecord(ctx->ev_side, ctx->side_stream) != cudaSuccess)
                st = md_fail(ctx, MD_ERR_CUDA, "cudaEventRecord on the side stream failed");
            ctx->stream = main_stream;
            MD_TRY(st);
        }
        MD_TRY(run_mixer(p, i));
        if (l.ff != MD_FF_NONE) MD_CUDA(ctx, cudaStreamWaitEvent(main_stream, ctx->ev_side, 0));
        next = update_after_parallel(s, b, i, p.rows, p.seqs);
    }
    if (ctx->stack_trace && !ctx->capturing) {
        next.x = b->x[0].as<float>(), next.x_out = b->x[1].as<float>();
        next.w[0] = s.w.final_norm, next.out[0] = b->h.p;
        MD_TRY(md_launch_parallel_glue(ctx, s.w.dtype, next));
        MD_TRY(keep_stream(p, s.layers.size() - 1, 1));
    }
    return MD_OK;
}

}  // namespace

int md_stack_layers(md_text_model* m, md_text_request* const* reqs, size_t seqs, size_t rows,
                    const unsigned long long* tokens_dev, bool decode, size_t pos0) {
    const Pass p = {m->ctx, *m->stack, reqs, seqs, rows, seqs * rows, decode, pos0, reqs[0]->stack};
    return m->stack->parallel ? parallel_layers(p, tokens_dev) : sandwich_layers(p, tokens_dev);
}

int md_stack_head(md_text_model* m, md_text_request* r0, size_t step_rows, const int* rows_dev, size_t n, float* logits,
                  unsigned long long* sampled, bool* keys) {
    md_ctx* ctx = m->ctx;
    const md_stack& s = *m->stack;
    md_stack_request* b = r0->stack;
    const size_t last = s.layers.size() - 1;
    if (s.parallel) {
        md_parallel_glue g = update_after_parallel(s, b, last, step_rows, 1);
        g.x = b->x[0].as<float>();
        g.w[0] = s.w.final_norm, g.out[0] = b->h.p;
        g.gather = rows_dev;
        g.rows = (int)n;
        MD_TRY(md_launch_parallel_glue(ctx, s.w.dtype, g));
    } else {
        md_glue g = update_after(s, b, last, s.layers[last].ff != MD_FF_NONE, step_rows, 1);
        g.x = b->x[final_x(s)].as<float>();
        g.x_out = nullptr;
        g.w_pre = s.w.final_norm;
        g.conv = nullptr;
        g.out = b->h.p;
        g.gather = rows_dev;
        g.rows = rows_dev ? (int)n : 1;
        g.seqs = rows_dev ? 1 : (int)n;
        MD_TRY(md_launch_glue(ctx, s.w.dtype, g));
    }
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
