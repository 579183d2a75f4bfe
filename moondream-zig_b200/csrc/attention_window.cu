// Grouped-query attention with a logarithmic distance bias, a sliding window with kept first tokens, values that are the
// keys, and one output gate per head (md_win_attn in stack.cuh).
//   append_keys_kernel      new key rows into the cache [kv_heads][max_seq][dim]
//   window_attention_kernel any element type and head size: one warp per (query, head), lanes over the head's dims
#include "stack.cuh"

namespace {

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

template <class T>
__global__ void __launch_bounds__(256)
append_keys_kernel(const __grid_constant__ md_win_attn p) {
    md_pdl_launch_dependents();
    md_pdl_wait();
    const int seq = blockIdx.y;
    const int pos0 = p.pos_dev[seq] ? *p.pos_dev[seq] : p.pos0;
    const int per = p.kv_heads * p.dim;
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long long)p.rows * per) return;
    const int t = (int)(i / per), c = (int)(i % per), g = c / p.dim, d = c % p.dim;
    const T* src = reinterpret_cast<const T*>(p.qkg) + (size_t)(seq * p.rows + t) * p.row_stride + p.heads * p.dim + c;
    reinterpret_cast<T*>(p.kc[seq])[((size_t)g * p.max_seq + pos0 + t) * p.dim + d] = *src;
}

constexpr int PER_LANE = 16;   // head sizes up to 512

template <class T>
__global__ void __launch_bounds__(128)
window_attention_kernel(const __grid_constant__ md_win_attn p) {
    md_pdl_launch_dependents();
    md_pdl_wait();
    const int lane = threadIdx.x & 31, seq = blockIdx.y;
    const int item = blockIdx.x * 4 + (threadIdx.x >> 5);
    if (item >= p.rows * p.heads) return;
    const int t = item / p.heads, h = item % p.heads, g = h / (p.heads / p.kv_heads);
    const int pos = (p.pos_dev[seq] ? *p.pos_dev[seq] : p.pos0) + t;
    const T* row = reinterpret_cast<const T*>(p.qkg) + (size_t)(seq * p.rows + t) * p.row_stride;
    const T* keys = reinterpret_cast<const T*>(p.kc[seq]) + (size_t)g * p.max_seq * p.dim;
    const float r1 = p.r1[h], r2 = p.r2[h];
    float q[PER_LANE], acc[PER_LANE];
#pragma unroll
    for (int i = 0; i < PER_LANE; ++i) {
        const int d = lane + 32 * i;
        q[i] = d < p.dim ? md_elem<T>::get(row[h * p.dim + d]) : 0.f;
        acc[i] = 0.f;
    }
    float m = -INFINITY, l = 0.f;
    auto visit = [&](int j) {
        const T* kr = keys + (size_t)j * p.dim;
        float k[PER_LANE], dot = 0.f;
#pragma unroll
        for (int i = 0; i < PER_LANE; ++i) {
            const int d = lane + 32 * i;
            k[i] = d < p.dim ? md_elem<T>::get(kr[d]) : 0.f;
            dot = fmaf(q[i], k[i], dot);
        }
        const float s = warp_sum(dot) * p.scale - r1 * log1pf(r2 * (float)(pos - j));
        const float mn = fmaxf(m, s), corr = m == -INFINITY ? 0.f : expf(m - mn), w = expf(s - mn);
        l = l * corr + w;
#pragma unroll
        for (int i = 0; i < PER_LANE; ++i) acc[i] = fmaf(acc[i], corr, w * k[i]);
        m = mn;
    };
    const int first = p.window > 0 ? max(0, pos - p.window + 1) : 0;
    for (int j = 0; j < min(p.keep_first, first); ++j) visit(j);
    for (int j = first; j <= pos; ++j) visit(j);
    const float gate = md_elem<T>::get(row[(p.heads + p.kv_heads) * p.dim + h]) / l;
    T* out = reinterpret_cast<T*>(p.out) + (size_t)(seq * p.rows + t) * p.heads * p.dim + h * p.dim;
#pragma unroll
    for (int i = 0; i < PER_LANE; ++i) {
        const int d = lane + 32 * i;
        if (d < p.dim) out[d] = md_elem<T>::put(acc[i] * gate);
    }
}

template <class T>
int launch(md_ctx* ctx, const md_win_attn& a) {
    const long long n = (long long)a.rows * a.kv_heads * a.dim;
    MD_TRY(md_launch_ex(ctx, append_keys_kernel<T>, dim3((unsigned)((n + 255) / 256), (unsigned)a.seqs), dim3(256), 0,
                        "append_keys_kernel", a));
    return md_launch_ex(ctx, window_attention_kernel<T>, dim3((unsigned)((a.rows * a.heads + 3) / 4), (unsigned)a.seqs),
                        dim3(128), 0, "window_attention_kernel", a);
}

}  // namespace

int md_launch_window_attention(md_ctx* ctx, int dtype, const md_win_attn& a, bool decode) {
    (void)decode;
    if (a.dim > 32 * PER_LANE) return md_fail(ctx, MD_ERR_UNSUPPORTED, "window attention: head size %d > %d", a.dim, 32 * PER_LANE);
    return dtype == MD_DTYPE_F32 ? launch<float>(ctx, a) : launch<__nv_bfloat16>(ctx, a);
}
