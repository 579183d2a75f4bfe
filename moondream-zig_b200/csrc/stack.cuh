// Internal declarations of the layer-stack decoders: text models described layer by layer (md_stack_weights of
// moondream_b200_model.h) instead of by one fixed layout.  The kernels are generic over the element type of weights and
// activations, T = __nv_bfloat16 (served) or float (every product in true 32-bit); the residual stream, norms, attention
// scores, recurrent states and routers are f32 in both.
#pragma once

#include <cuda_bf16.h>

#include "md_internal.cuh"

#include "../../include/moondream_b200_model.h"

constexpr int MD_STACK_MAX_SEQS = 8;     // requests advanced together by one step
constexpr int MD_STACK_MAX_TAPS = 8;
constexpr int MD_GROUP_ROWS = 128;       // an expert's rows in the sorted buffers start at a multiple of this

// ---- linear layers: C[M,N] = act(A[M,K] . W[N,K]^T + bias) --------------------------------------------------
struct md_lin {
    const float* bias = nullptr;     // [N] or null
    int silu_cols = 0;               // columns < silu_cols go through silu
    int sigmoid_from = 1 << 30;      // columns >= sigmoid_from go through the logistic function
    // glu != 0: W's rows are gate and up rows in alternating blocks of 32 (MD_GLU_BLOCK) and C[M, N/2] = act(gate) * up
    int glu = 0;                     // MD_ACT_*
    float glu_limit = 0.f, glu_alpha = 0.f;   // MD_ACT_CLAMPED (md_gated)
    float* out_f32 = nullptr;        // write f32 sums here instead of T to C
    unsigned long long* amax = nullptr;   // [M] running maximum of md_argmax_key over each row (bfloat16, M <= 8; zero before)
    // rows sorted by expert: row block b (128 rows) belongs to expert tile_expert[b], whose matrix is W + e * N * K;
    // only the first *n_blocks blocks are computed
    const int* tile_expert = nullptr;
    const int* n_blocks = nullptr;
    int n_experts = 0;
};
constexpr int MD_GLU_BLOCK = 32;
// bfloat16 kernels behind md_linear (weights [N, K])
int md_launch_gemm_tc_lin(md_ctx* ctx, const void* a, const void* b, void* c, size_t M, size_t N, size_t K, const md_lin& lin);
int md_launch_gemm_pair_lin(md_ctx* ctx, const void* a, const void* b, void* c, size_t M, size_t N, size_t K, const md_lin& lin);
int md_launch_gemm_skinny_lin(md_ctx* ctx, const void* a, const void* b, void* c, size_t M, size_t N, size_t K, const md_lin& lin);
int md_launch_gemv_lin(md_ctx* ctx, const void* a, const void* b, void* c, size_t M, size_t N, size_t K, const md_lin& lin);
inline bool md_gemv_lin_supported(const void* a, const void* w, size_t K) {
    return (K % 8) == 0 && ((reinterpret_cast<uintptr_t>(a) | reinterpret_cast<uintptr_t>(w)) & 15) == 0;
}
int md_make_map_2d_bf16(md_ctx* ctx, CUtensorMap* map, const void* ptr, uint64_t inner, uint64_t outer, uint32_t box_inner,
                        uint32_t box_outer, bool swizzle_64);
int md_linear(md_ctx* ctx, int dtype, const void* a, const void* w, void* c, size_t M, size_t N, size_t K, const md_lin& ep);

// ---- residual + norms + causal convolution ---------------------------------------------------------------
// For every row t of a sequence:
//   x_out[t] = x[t] + mult * rms_norm(y[t]; w_post)             (y == null: x_out = x; tokens != null: x = embed[token])
//   n[t]     = rms_norm(x_out[t]; w_pre)
//   out[t]   = n[t] + sum_j conv[j] * n[t - taps + 1 + j]       (conv == null: out = n)
// The convolution's last taps - 1 inputs live in `state` between calls: two copies of [taps - 1][width] f32, of which
// *state_slot (device memory) names the current one.  A decode step (rows == 1) updates it in place; a prompt's portion
// reads it and writes the other one, since different blocks read the start and write the end, and whoever ends the step
// flips *state_slot.
struct md_glue {
    int width = 0, rows = 0, taps = 0;      // rows per sequence
    float eps = 0.f, mult = 0.f;
    const float* x = nullptr;               // [seqs * rows, width]
    float* x_out = nullptr;                 // must differ from x when rows > 1
    const void* embed = nullptr;            // [vocab, width] T
    const unsigned long long* tokens = nullptr;
    int vocab = 0;
    // the sublayer's output, one of: f32 rows, T rows, or T rows of the expert-sorted buffer
    const float* y_f32 = nullptr;
    const void* y = nullptr;
    const float* w_post = nullptr;
    // y is scaled per row by 1 / sqrt(sum(ssq) / ssq_n + eps) (the norm ahead of the output projection, applied after it)
    const float* ssq = nullptr;             // [rows, ssq_parts]
    int ssq_parts = 0, ssq_n = 0;
    // mixture of experts: y of row t = sum_k score[t][k] * y[slot[t][k]]
    const int* slot = nullptr;              // [rows, top]: place in the sorted rows
    const float* score = nullptr;
    int top = 0;
    const float* w_pre = nullptr;
    const float* conv = nullptr;            // [taps][width]
    void* out = nullptr;                    // [seqs * rows, width] T
    const int* gather = nullptr;            // rows to take (final norm of the wanted rows): x row = gather[i], no x_out
    int seqs = 1;
    float* state[MD_STACK_MAX_SEQS] = {};
    const int* state_slot[MD_STACK_MAX_SEQS] = {};
};
int md_launch_glue(md_ctx* ctx, int dtype, const md_glue& g);

// The same place in a layer whose two sublayers read the same residual row (MD_LAYER_PARALLEL).  For every row:
//   x_out = x + sum_b scale_b * y_b      (b = the sublayers that ran; tokens != null: x = embed[token])
//   n     = x_out / sqrt(mean(x_out^2) + eps);  out[o] = n * w[o]   for up to two outputs
struct md_branch {
    const float* y_f32 = nullptr;           // the sublayer's output, as in md_glue: f32 rows, T rows,
    const void* y = nullptr;
    const int* slot = nullptr;              //   or T rows of the expert-sorted buffer: sum_k score[t][k] * y[slot[t][k]]
    const float* score = nullptr;
    int top = 0;
    const float* scale = nullptr;           // [width]
};
struct md_parallel_glue {
    int width = 0, rows = 0;                // rows of all sequences
    float eps = 0.f;
    const float* x = nullptr;
    float* x_out = nullptr;                 // may be x
    const void* embed = nullptr;
    const unsigned long long* tokens = nullptr;
    int vocab = 0;
    md_branch b[2];
    const float* w[2] = {};
    void* out[2] = {};                      // [rows, width] T
    const int* gather = nullptr;            // as in md_glue
};
int md_launch_parallel_glue(md_ctx* ctx, int dtype, const md_parallel_glue& g);

// ---- attention: distance bias, sliding window with kept first keys, values = keys, gated heads -------------
struct md_win_attn {
    int heads = 0, kv_heads = 0, dim = 0;
    float scale = 0.f;
    int window = 0, keep_first = 0;         // window <= 0: unlimited
    const float *r1 = nullptr, *r2 = nullptr;
    const void* qkg = nullptr;              // rows [q: heads * dim | k: kv_heads * dim | gate: heads (logistic applied)]
    int row_stride = 0;
    void* out = nullptr;                    // [rows, heads * dim] T
    int rows = 0;                           // per sequence
    size_t max_seq = 0;
    int seqs = 1;
    void* kc[MD_STACK_MAX_SEQS] = {};       // [kv_heads][max_seq][dim] T
    const int* pos_dev[MD_STACK_MAX_SEQS] = {};   // decode: position of the new token
    int pos0 = 0;                           // prefill: position of row 0
};
int md_launch_window_attention(md_ctx* ctx, int dtype, const md_win_attn& a, bool decode);

// ---- latent attention: keys and values of all heads are linear maps of one cached latent per token -----------
// Per token: cq = rms(in[0 .. q_rank); q_norm), c = rms(in[q_rank .. + kv_rank); kv_norm), kr = rotated in[.. + rot).  Cached:
// c and kr.  Head h: q = w_uq cq, k = w_uk c, v = w_uv c; score(i, j) = scale * (q . k_j + rotated q . kr_j); softmax whose
// denominator also holds exp(sink[h]).
struct md_latent {
    int heads = 0, dim = 0, rot = 0, vdim = 0, q_rank = 0, kv_rank = 0;
    float scale = 0.f, eps = 0.f;
    int window = 0;                         // <= 0: unlimited
    const float *q_norm = nullptr, *kv_norm = nullptr, *sink = nullptr;
    const float* rope = nullptr;            // [max_seq][rot / 2] (cos, sin)
    const void* w_uq = nullptr;             // [heads * (dim + rot), q_rank]: per head [dim | rot]
    const void* w_ukv = nullptr;            // [heads * dim (keys) + heads * vdim (values), kv_rank]
    const void* w_ukt = nullptr;            // [heads][kv_rank][dim] (bfloat16 decoding; null: not available)
    const void* in = nullptr;               // [rows of all sequences, row_stride] T
    int row_stride = 0;
    void *cq = nullptr, *q = nullptr;       // [rows, q_rank], [rows, heads * (dim + rot)] T
    void* out = nullptr;                    // [rows, heads * vdim] T
    int rows = 0, seqs = 1;                 // rows per sequence
    size_t max_seq = 0;
    void* cc[MD_STACK_MAX_SEQS] = {};       // [max_seq][kv_rank] T
    void* kr[MD_STACK_MAX_SEQS] = {};       // [max_seq][rot] T
    const int* pos_dev[MD_STACK_MAX_SEQS] = {};   // decode: position of the new token
    int pos0 = 0;                           // prefill: position of row 0
    // prompts in bfloat16: keys and values of every visible token, [md_latent_keys(..)][heads * (dim + vdim)]
    void* kv = nullptr;
    void* qa = nullptr;                     // bfloat16 decoding: queries in the latent space [seqs][heads][kv_rank + rot]
};
// tokens whose keys a portion of `rows` rows can see (itself included)
inline size_t md_latent_keys(size_t rows, size_t window, size_t max_seq) {
    return window > 0 && rows + window - 1 < max_seq ? rows + window - 1 : max_seq;
}
// whether a portion of `rows` rows of one sequence takes the tensor-core prompt kernel (and so needs md_latent::kv)
bool md_latent_expands(int dtype, const md_latent& a);
int md_launch_latent_attention(md_ctx* ctx, int dtype, const md_latent& a, bool decode);
// the prompt kernel on tcgen05 (bfloat16; head sizes it cannot hold take latent_prefill_kernel)
bool md_latent_tc_supported(const md_latent& a);
int md_launch_latent_tc(md_ctx* ctx, const md_latent& a, int key0);
// (cos, sin) of pos * base^(-2 i / dims) for pos < rows, i < dims / 2; angles in f64
int md_launch_rotation_table(md_ctx* ctx, float* table, size_t rows, size_t dims, float base);

// ---- linear attention with per-head decay ----------------------------------------------------------------
struct md_lightning {
    int heads = 0, dim = 0, vdim = 0;
    const float* decay = nullptr;           // [heads] device
    const float* norm_w = nullptr;          // [heads * vdim]
    const void* qkvg = nullptr;             // rows [q | k | v (all through silu) | g (logistic applied)]
    int row_stride = 0;
    void* out = nullptr;                    // [rows, heads * vdim] T: o * norm_w * gate, not yet divided by its rms
    float* ssq = nullptr;                   // [rows, ssq_parts]: sums of o^2
    int ssq_parts = 0;
    int rows = 0, seqs = 1;
    float* state[MD_STACK_MAX_SEQS] = {};   // [heads][dim][vdim] f32
};
// number of ssq entries a row has for these sizes
int md_lightning_ssq_parts(int heads, int vdim);
int md_launch_lightning(md_ctx* ctx, int dtype, const md_lightning& l, bool decode);

// ---- mixture of experts --------------------------------------------------------------------------------------
struct md_moe {
    int width = 0, experts = 0, top = 0, ff_pad = 0, act = 0;
    float limit = 0.f, alpha = 0.f;          // of the activation (md_gated)
    int router_kind = 0;                     // MD_ROUTER_*
    const void *router = nullptr, *w_gu = nullptr, *w_down = nullptr;   // [E (+ 1), W], [E, 2 ff_pad, W], [E, W, ff_pad]
    // shared expert (shared_pad > 0): runs for every token, weighted with the logistic of the router's row E
    int shared_pad = 0;
    float shared_limit = 0.f;
    const void *shared_gu = nullptr, *shared_down = nullptr;            // [2 shared_pad, W], [W, shared_pad]
    int choices() const { return top + (shared_pad > 0 ? 1 : 0); }      // entries of a token in score and slot
};
struct md_moe_buffers {
    float* score = nullptr;       // [rows, choices]
    int* slot = nullptr;          // [rows, choices]
    int *sel = nullptr, *rank = nullptr;                      // [rows, top]
    int *count = nullptr;         // [experts]
    int *tile_expert = nullptr, *n_blocks = nullptr;
    // sorted rows; act also takes 8 rows of shared_pad, ys also the shared expert's row of every token
    void *xs = nullptr, *act = nullptr, *ys = nullptr;
    void* shared_act = nullptr;   // [rows, shared_pad]
    float* y_f32 = nullptr;       // [rows, width], rows <= 8
    float* route = nullptr;       // md_moe_route_floats(experts), zeroed once
};
inline size_t md_moe_route_floats(size_t experts) { return 17 * (experts + 1) + 16; }
size_t md_moe_sorted_rows(size_t rows, int experts, int top);   // capacity of the sorted buffers
// true: md_launch_moe leaves a token's outputs in the sorted rows (slot, score, ys); false: their sum in y_f32
bool md_moe_sorted(int dtype, size_t width, size_t rows);
int md_launch_moe(md_ctx* ctx, int dtype, const md_moe& m, const void* h, size_t rows, const md_moe_buffers& b);

int md_launch_argmax_f32(md_ctx* ctx, const float* x, size_t n, size_t stride, size_t rows, unsigned long long* idx_dev);

#ifdef __CUDACC__
// An order-preserving image of the value above the complement of the index: the largest key is the first largest value.
__device__ __forceinline__ unsigned long long md_argmax_key(float v, uint32_t i) {
    const uint32_t b = __float_as_uint(v);
    return ((unsigned long long)((b & 0x80000000u) ? ~b : (b | 0x80000000u)) << 32) | (0xFFFFFFFFu - i);
}
template <class T> struct md_elem;
template <> struct md_elem<__nv_bfloat16> {
    static __device__ __forceinline__ float get(__nv_bfloat16 v) { return __bfloat162float(v); }
    static __device__ __forceinline__ __nv_bfloat16 put(float v) { return __float2bfloat16_rn(v); }
};
template <> struct md_elem<float> {
    static __device__ __forceinline__ float get(float v) { return v; }
    static __device__ __forceinline__ float put(float v) { return v; }
};
__device__ __forceinline__ float md_logistic(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float md_silu(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float md_gelu_tanh(float z) {
    return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
__device__ __forceinline__ float md_act(int act, float z) { return act == MD_ACT_SILU ? md_silu(z) : md_gelu_tanh(z); }
// gate and up of a gated feed-forward
__device__ __forceinline__ float md_gated(int act, float limit, float alpha, float g, float u) {
    if (act == MD_ACT_CLAMPED) {
        g = fminf(g, limit);
        u = fminf(fmaxf(u, -limit), limit);
        return g * md_logistic(alpha * g) * (u + 1.f);
    }
    return md_act(act, g) * u;
}
// column activation of md_lin
__device__ __forceinline__ float md_lin_col(float v, int n, int silu_cols, int sigmoid_from) {
    if (n < silu_cols) return md_silu(v);
    if (n >= sigmoid_from) return md_logistic(v);
    return v;
}
template <class T> __device__ __forceinline__ void md_load4(const T* p, float (&f)[4]);
template <> __device__ __forceinline__ void md_load4<float>(const float* p, float (&f)[4]) {
    const float4 v = __ldcg(reinterpret_cast<const float4*>(p));
    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
}
template <> __device__ __forceinline__ void md_load4<__nv_bfloat16>(const __nv_bfloat16* p, float (&f)[4]) {
    const uint2 u = __ldcg(reinterpret_cast<const uint2*>(p));
    f[0] = __uint_as_float(u.x << 16); f[1] = __uint_as_float(u.x & 0xffff0000u);
    f[2] = __uint_as_float(u.y << 16); f[3] = __uint_as_float(u.y & 0xffff0000u);
}
__device__ __forceinline__ uint32_t md_pack_bf16(float lo, float hi) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&h);
}
template <class T> __device__ __forceinline__ void md_store4(T* p, const float (&f)[4]);
template <> __device__ __forceinline__ void md_store4<float>(float* p, const float (&f)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
}
template <> __device__ __forceinline__ void md_store4<__nv_bfloat16>(__nv_bfloat16* p, const float (&f)[4]) {
    *reinterpret_cast<uint2*>(p) = make_uint2(md_pack_bf16(f[0], f[1]), md_pack_bf16(f[2], f[3]));
}
#endif
