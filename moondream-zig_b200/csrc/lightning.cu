// Linear attention with a per-head decay (md_lightning in stack.cuh).
//   lightning_scan_kernel  any element type, head size and length: a block owns 32 value columns of one head of one
//                          sequence, keeps its [dim][32] part of the state in shared memory (f32) and walks the tokens.
// The RMS norm over the concatenated heads is a scalar per row ahead of a linear map, so the kernels only leave the sums
// of squares; whoever reads the output projection divides (md_glue::ssq).
#include "stack.cuh"

namespace {

constexpr int VB = 32;    // value columns per block

template <class T>
__global__ void __launch_bounds__(256)
lightning_scan_kernel(const __grid_constant__ md_lightning p) {
    extern __shared__ float sm[];
    const int dim = p.dim;
    float *S = sm, *qs = sm + dim * VB, *ks = qs + dim, *red = ks + dim;   // red [8][32]
    md_pdl_launch_dependents();
    md_pdl_wait();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int vb = blockIdx.x, h = blockIdx.y, seq = blockIdx.z;
    const int v0 = vb * VB, v = v0 + lane;
    const bool live = v < p.vdim;
    float* state = p.state[seq] + (size_t)h * dim * p.vdim;
    for (int d = warp; d < dim; d += 8) S[d * VB + lane] = live ? state[(size_t)d * p.vdim + v] : 0.f;
    const float decay = p.decay[h];
    const int Q = 0, Kc = p.heads * dim, Vc = 2 * p.heads * dim, Gc = Vc + p.heads * p.vdim;
    for (int t = 0; t < p.rows; ++t) {
        const size_t row = (size_t)seq * p.rows + t;
        const T* r = reinterpret_cast<const T*>(p.qkvg) + row * p.row_stride;
        __syncthreads();
        for (int d = tid; d < dim; d += 256) {
            qs[d] = md_elem<T>::get(r[Q + h * dim + d]);
            ks[d] = md_elem<T>::get(r[Kc + h * dim + d]);
        }
        const float vv = live ? md_elem<T>::get(r[Vc + h * p.vdim + v]) : 0.f;
        __syncthreads();
        float o = 0.f;
        for (int d = warp; d < dim; d += 8) {
            const float s = fmaf(decay, S[d * VB + lane], ks[d] * vv);
            S[d * VB + lane] = s;
            o = fmaf(qs[d], s, o);
        }
        red[warp * 32 + lane] = o;
        __syncthreads();
        if (warp == 0) {
            o = 0.f;
#pragma unroll
            for (int w = 0; w < 8; ++w) o += red[w * 32 + lane];
            float sq = live ? o * o : 0.f;
#pragma unroll
            for (int i = 16; i; i >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, i);
            if (lane == 0) p.ssq[row * p.ssq_parts + h * gridDim.x + vb] = sq;
            if (live) {
                const int c = h * p.vdim + v;
                reinterpret_cast<T*>(p.out)[row * (p.heads * p.vdim) + c] =
                    md_elem<T>::put(o * p.norm_w[c] * md_elem<T>::get(r[Gc + c]));
            }
        }
    }
    __syncthreads();
    if (live)
        for (int d = warp; d < dim; d += 8) state[(size_t)d * p.vdim + v] = S[d * VB + lane];
}

template <class T>
int launch_scan(md_ctx* ctx, const md_lightning& l) {
    const size_t smem = ((size_t)l.dim * VB + 2 * l.dim + 256) * sizeof(float);
    if (smem > 220 * 1024) return md_fail(ctx, MD_ERR_UNSUPPORTED, "lightning: head size %d", l.dim);
    if (smem > 48 * 1024)
        MD_CUDA(ctx, cudaFuncSetAttribute(lightning_scan_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
    return md_launch_ex(ctx, lightning_scan_kernel<T>, dim3((unsigned)((l.vdim + VB - 1) / VB), (unsigned)l.heads, (unsigned)l.seqs),
                        dim3(256), smem, "lightning_scan_kernel", l);
}

}  // namespace

int md_lightning_ssq_parts(int heads, int vdim) { return heads * ((vdim + VB - 1) / VB); }

int md_launch_lightning(md_ctx* ctx, int dtype, const md_lightning& l, bool decode) {
    (void)decode;
    return dtype == MD_DTYPE_F32 ? launch_scan<float>(ctx, l) : launch_scan<__nv_bfloat16>(ctx, l);
}
