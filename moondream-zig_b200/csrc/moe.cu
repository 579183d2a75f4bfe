// Mixture of experts with independent logistic scores (md_moe in stack.cuh).
//   moe_router_kernel   scores and top choice per token (f32), and each (token, expert) pair's rank within its expert
//   moe_permute_kernel  rows sorted by expert, every expert's rows starting at a multiple of 128
// then the two expert products run as grouped products over the sorted rows, and the weighted sum of a token's experts
// is taken where the residual is updated (md_glue::slot).
#include "stack.cuh"

namespace {

constexpr int MAX_EXPERTS = 512, MAX_TOP = 32;

// one warp per token
template <class T>
__global__ void __launch_bounds__(128)
moe_router_kernel(const T* __restrict__ h, const T* __restrict__ router, int rows, int W, int E, int top, float* score,
                  int* sel, int* rank, int* count) {
    __shared__ float s_all[4][MAX_EXPERTS];
    md_pdl_launch_dependents();
    md_pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x * 4 + warp;
    if (t >= rows) return;
    float* s = s_all[warp];
    const T* hr = h + (size_t)t * W;
    for (int e = 0; e < E; ++e) {
        const T* wr = router + (size_t)e * W;
        float z = 0.f;
        for (int c = lane; c < W; c += 32) z = fmaf(md_elem<T>::get(hr[c]), md_elem<T>::get(wr[c]), z);
#pragma unroll
        for (int o = 16; o; o >>= 1) z += __shfl_xor_sync(0xffffffffu, z, o);
        if (lane == 0) s[e] = md_logistic(z);
    }
    __syncwarp();
    for (int k = 0; k < top; ++k) {
        float best = -1.f;
        int bi = 0;
        for (int e = lane; e < E; e += 32)
            if (s[e] > best) { best = s[e]; bi = e; }
#pragma unroll
        for (int o = 16; o; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (ob > best || (ob == best && oi < bi)) { best = ob; bi = oi; }
        }
        if (lane == 0) {
            score[(size_t)t * top + k] = best;
            sel[(size_t)t * top + k] = bi;
            rank[(size_t)t * top + k] = atomicAdd(count + bi, 1);
            s[bi] = -2.f;
        }
        __syncwarp();
    }
}

template <class T>
__global__ void __launch_bounds__(256)
moe_permute_kernel(const T* __restrict__ h, int W, int E, int top, const int* __restrict__ sel, const int* __restrict__ rank,
                   const int* __restrict__ count, int* slot, int* tile_expert, int* n_blocks, T* __restrict__ xs) {
    __shared__ int first[MAX_EXPERTS + 1];   // first row block of every expert
    md_pdl_launch_dependents();
    md_pdl_wait();
    if (threadIdx.x < 32) {
        int run = 0;
        for (int e0 = 0; e0 < E; e0 += 32) {
            const int e = e0 + threadIdx.x;
            const int mine = e < E ? (count[e] + MD_GROUP_ROWS - 1) / MD_GROUP_ROWS : 0;
            int inc = mine;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int v = __shfl_up_sync(0xffffffffu, inc, o);
                if ((int)threadIdx.x >= o) inc += v;
            }
            if (e < E) first[e] = run + inc - mine;
            run += __shfl_sync(0xffffffffu, inc, 31);
        }
        if (threadIdx.x == 0) first[E] = run;
    }
    __syncthreads();
    const int t = blockIdx.x;
    if (t == 0) {
        for (int e = threadIdx.x; e < E; e += blockDim.x)
            for (int b = first[e]; b < first[e + 1]; ++b) tile_expert[b] = e;
        if (threadIdx.x == 0) *n_blocks = first[E];
    }
    const T* src = h + (size_t)t * W;
    for (int k = 0; k < top; ++k) {
        const int e = sel[(size_t)t * top + k], row = first[e] * MD_GROUP_ROWS + rank[(size_t)t * top + k];
        if (threadIdx.x == 0) slot[(size_t)t * top + k] = row;
        T* dst = xs + (size_t)row * W;
        if ((W % 4) == 0) {
            for (int c = threadIdx.x * 4; c < W; c += blockDim.x * 4) {
                float f[4];
                md_load4<T>(src + c, f);
                md_store4<T>(dst + c, f);
            }
        } else {
            for (int c = threadIdx.x; c < W; c += blockDim.x) dst[c] = src[c];
        }
    }
}

template <class T>
int launch_sorted(md_ctx* ctx, int dtype, const md_moe& m, const void* h, size_t rows, const md_moe_buffers& b) {
    MD_CUDA(ctx, cudaMemsetAsync(b.count, 0, m.experts * sizeof(int), ctx->stream));
    MD_TRY(md_launch_ex(ctx, moe_router_kernel<T>, dim3((unsigned)((rows + 3) / 4)), dim3(128), 0, "moe_router_kernel",
                        reinterpret_cast<const T*>(h), reinterpret_cast<const T*>(m.router), (int)rows, m.width, m.experts,
                        m.top, b.score, b.sel, b.rank, b.count));
    MD_TRY(md_launch_ex(ctx, moe_permute_kernel<T>, dim3((unsigned)rows), dim3(256), 0, "moe_permute_kernel",
                        reinterpret_cast<const T*>(h), m.width, m.experts, m.top, b.sel, b.rank, b.count, b.slot,
                        b.tile_expert, b.n_blocks, reinterpret_cast<T*>(b.xs)));
    const size_t cap = md_moe_sorted_rows(rows, m.experts, m.top);
    md_lin up;
    up.glu = m.act;
    up.tile_expert = b.tile_expert;
    up.n_blocks = b.n_blocks;
    up.n_experts = m.experts;
    MD_TRY(md_linear(ctx, dtype, b.xs, m.w_gu, b.act, cap, 2 * (size_t)m.ff_pad, m.width, up));
    md_lin down = up;
    down.glu = 0;
    return md_linear(ctx, dtype, b.act, m.w_down, b.ys, cap, m.width, m.ff_pad, down);
}

}  // namespace

bool md_moe_sorted(int dtype, size_t rows) {
    (void)dtype, (void)rows;
    return true;
}

size_t md_moe_sorted_rows(size_t rows, int experts, int top) {
    const size_t pairs = rows * top, used = pairs < (size_t)experts ? pairs : (size_t)experts;
    // every expert with a row wastes at most GROUP - 1 rows
    return (pairs + used * (MD_GROUP_ROWS - 1) + MD_GROUP_ROWS - 1) / MD_GROUP_ROWS * MD_GROUP_ROWS;
}

int md_launch_moe(md_ctx* ctx, int dtype, const md_moe& m, const void* h, size_t rows, const md_moe_buffers& b) {
    if (m.experts > MAX_EXPERTS || m.top > MAX_TOP || m.top > m.experts)
        return md_fail(ctx, MD_ERR_UNSUPPORTED, "mixture of experts: %d experts, %d per token", m.experts, m.top);
    return dtype == MD_DTYPE_F32 ? launch_sorted<float>(ctx, dtype, m, h, rows, b)
                                 : launch_sorted<__nv_bfloat16>(ctx, dtype, m, h, rows, b);
}
