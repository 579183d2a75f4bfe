// Linear layers of the layer-stack decoders: md_linear picks the kernel (the bfloat16 forms of the GEMV, the skinny GEMM
// and the tcgen05 GEMMs, by the rules of the f16 dispatch), and gemm_plain_kernel is the one that takes any
// shape and either element type (the true 32-bit products, and bfloat16 shapes whose rows TMA or 16-byte loads cannot
// address): 64 x 64 tiles, f32 FMA.
#include "stack.cuh"

namespace {

constexpr int TILE = 64, KB = 16;

template <class T>
__global__ void __launch_bounds__(256)
gemm_plain_kernel(const T* __restrict__ A, const T* __restrict__ Wt, T* __restrict__ C, int M, int N, int K, md_lin ep) {
    __shared__ float As[KB][TILE + 4], Bs[KB][TILE + 4];
    md_pdl_launch_dependents();
    md_pdl_wait();
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int m0 = blockIdx.y * TILE, n0 = blockIdx.x * TILE;
    if (ep.tile_expert) {
        const int block = m0 / MD_GROUP_ROWS;
        if (block >= *ep.n_blocks) return;
        Wt += (size_t)ep.tile_expert[block] * N * K;
    }
    // a thread's columns: two of the tile's first half and the two 32 further on (a gate and its up column)
    float acc[4][4] = {};
    for (int k0 = 0; k0 < K; k0 += KB) {
        for (int i = tid; i < TILE * KB; i += 256) {
            const int r = i / KB, k = i % KB;
            As[k][r] = (m0 + r < M && k0 + k < K) ? md_elem<T>::get(A[(size_t)(m0 + r) * K + k0 + k]) : 0.f;
            Bs[k][r] = (n0 + r < N && k0 + k < K) ? md_elem<T>::get(Wt[(size_t)(n0 + r) * K + k0 + k]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < KB; ++k) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) a[i] = As[k][ty * 4 + i];
#pragma unroll
            for (int j = 0; j < 4; ++j) b[j] = Bs[k][tx * 2 + (j & 1) + (j >> 1) * 32];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int m = m0 + ty * 4 + i;
        if (m >= M) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int n = n0 + tx * 2 + (j & 1) + (j >> 1) * 32;
            if (n >= N) continue;
            if (ep.glu) {
                if (j < 2) C[(size_t)m * (N / 2) + n0 / 2 + tx * 2 + j] = 
                    md_elem<T>::put(md_gated(ep.glu, ep.glu_limit, ep.glu_alpha, acc[i][j], acc[i][j + 2]));
                continue;
            }
            float v = acc[i][j];
            if (ep.bias) v += ep.bias[n];
            v = md_lin_col(v, n, ep.silu_cols, ep.sigmoid_from);
            if (ep.out_f32) ep.out_f32[(size_t)m * N + n] = v;
            else C[(size_t)m * N + n] = md_elem<T>::put(v);
        }
    }
}

template <class T>
int launch_plain(md_ctx* ctx, const void* a, const void* w, void* c, size_t M, size_t N, size_t K, const md_lin& ep) {
    return md_launch_ex(ctx, gemm_plain_kernel<T>, dim3((unsigned)((N + TILE - 1) / TILE), (unsigned)((M + TILE - 1) / TILE)),
                        dim3(256), 0, "gemm_plain_kernel", reinterpret_cast<const T*>(a), reinterpret_cast<const T*>(w),
                        reinterpret_cast<T*>(c), (int)M, (int)N, (int)K, ep);
}

}  // namespace

int md_linear(md_ctx* ctx, int dtype, const void* a, const void* w, void* c, size_t M, size_t N, size_t K, const md_lin& ep) {
    if (M == 0 || N == 0) return MD_OK;
    if (ep.glu && (N % (2 * MD_GLU_BLOCK)) != 0) return md_fail(ctx, MD_ERR_INVALID_ARG, "md_linear: gate / up rows must come in blocks");
    if (dtype == MD_DTYPE_F32) return launch_plain<float>(ctx, a, w, c, M, N, K, ep);
    const uintptr_t align = reinterpret_cast<uintptr_t>(a) | reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(c);
    if ((ctx->gemm_mode != 1 || ep.amax) && (K % 8) == 0 && (align & 15) == 0) {
        if (!ep.tile_expert && (M <= 8 || ep.out_f32)) {
            // f32 results of many rows (the head over the wanted rows of a prompt): eight rows at a time
            for (size_t m = 0; m < M; m += 8) {
                md_lin part = ep;
                if (ep.out_f32) part.out_f32 = ep.out_f32 + m * N;
                MD_TRY(md_launch_gemv_lin(ctx, reinterpret_cast<const __nv_bfloat16*>(a) + m * K, w, c, M - m < 8 ? M - m : 8, N, K, part));
            }
            return MD_OK;
        }
        if ((N % 8) == 0 && !ep.out_f32) {
            if (!ep.tile_expert && ctx->skinny && md_gemm_skinny_supported(a, w, c, M, N, K))
                return md_launch_gemm_skinny_lin(ctx, a, w, c, M, N, K, ep);
            return md_launch_gemm_tc_lin(ctx, a, w, c, M, N, K, ep);
        }
    }
    return launch_plain<__nv_bfloat16>(ctx, a, w, c, M, N, K, ep);
}
