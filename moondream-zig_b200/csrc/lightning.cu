// Linear attention with a per-head decay (md_lightning in stack.cuh).
//   lightning_scan_kernel  any element type, head size and length: a block owns 32 value columns of one head of one
//                          sequence, keeps its [dim][32] part of the state in shared memory (f32) and walks the tokens.
//   lightning_step_kernel  one token per sequence (decode), any element type: the same split, the state in registers and
//                          requested before the dependency wait.
// bfloat16 prompts in chunks of 64 tokens on tensor cores.  Within a chunk that starts from state S (lambda = decay):
//     o_i = lambda^(i+1) S^T q_i + sum_(j <= i) lambda^(i-j) (q_i . k_j) v_j
//     S  <- lambda^len S + sum_j lambda^(len-1-j) k_j v_j^T
// The f32 factors of a product (S, the decayed scores, the decayed values) enter as two bfloat16 terms each
// (mma_bf16.cuh); q, k, v are bfloat16 as they are, sums and the state are f32.
//   lightning_chunk_kernel<OUT>  one head and one segment of chunks per block.  OUT: outputs, and the final state from the
//                          last segment.  Otherwise only the segment's own contribution to the state.
//   lightning_carry_kernel  the state each segment starts from, out of the segments' contributions.
// A prompt short enough for one segment takes the first kernel alone.
// The RMS norm over the concatenated heads is a scalar per row ahead of a linear map, so the kernels only leave the sums
// of squares; whoever reads the output projection divides (md_glue::ssq).
#include "mma_bf16.cuh"

namespace {

constexpr int VB = 32;    // value columns per block

template <class T>
__global__ void __launch_bounds__(256)
lightning_scan_kernel(const __grid_constant__ md_lightning p) {
    extern __shared__ __align__(16) unsigned char sm[];
    const int dim = p.dim;
    float *S = reinterpret_cast<float*>(sm), *qs = S + dim * VB, *ks = qs + dim, *red = ks + dim;   // red [8][32]
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

// rows of a warp: d = warp + 8 i, i < N
template <class T, int N>
__global__ void __launch_bounds__(256)
lightning_step_kernel(const __grid_constant__ md_lightning p) {
    __shared__ float red[8][32];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, dim = p.dim;
    const int vb = blockIdx.x, h = blockIdx.y, seq = blockIdx.z, v = vb * VB + lane;
    const bool live = v < p.vdim;
    md_pdl_launch_dependents();
    float* state = p.state[seq] + (size_t)h * dim * p.vdim + v;
    const float decay = p.decay[h];
    const int c = h * p.vdim + v;
    const float nw = live ? p.norm_w[c] : 0.f;
    float S[N];
#pragma unroll
    for (int i = 0; i < N; ++i) {
        const int d = warp + 8 * i;
        S[i] = live && d < dim ? __ldcg(state + (size_t)d * p.vdim) : 0.f;
    }
    md_pdl_wait();
    const T* r = reinterpret_cast<const T*>(p.qkvg) + (size_t)seq * p.row_stride;
    const int Kc = p.heads * dim, Vc = 2 * p.heads * dim, Gc = Vc + p.heads * p.vdim;
    const float vv = live ? md_elem<T>::get(__ldcg(r + Vc + c)) : 0.f;
    const float gate = live ? md_elem<T>::get(__ldcg(r + Gc + c)) : 0.f;
    float k[N], q[N], o = 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i) {
        const int d = warp + 8 * i;
        k[i] = d < dim ? md_elem<T>::get(__ldcg(r + Kc + h * dim + d)) : 0.f;
        q[i] = d < dim ? md_elem<T>::get(__ldcg(r + h * dim + d)) : 0.f;
    }
#pragma unroll
    for (int i = 0; i < N; ++i) {
        const int d = warp + 8 * i;
        S[i] = fmaf(decay, S[i], k[i] * vv);
        if (live && d < dim) state[(size_t)d * p.vdim] = S[i];
        o = fmaf(q[i], S[i], o);
    }
    red[warp][lane] = o;
    __syncthreads();
    if (warp == 0) {
        o = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) o += red[w][lane];
        float sq = live ? o * o : 0.f;
#pragma unroll
        for (int i = 16; i; i >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, i);
        if (lane == 0) p.ssq[(size_t)seq * p.ssq_parts + h * gridDim.x + vb] = sq;
        if (live) reinterpret_cast<T*>(p.out)[(size_t)seq * (p.heads * p.vdim) + c] = md_elem<T>::put(o * nw * gate);
    }
}

template <class T>
int launch_step(md_ctx* ctx, const md_lightning& l) {
    const dim3 grid((unsigned)((l.vdim + VB - 1) / VB), (unsigned)l.heads, (unsigned)l.seqs);
    if (l.dim <= 64) return md_launch_ex(ctx, lightning_step_kernel<T, 8>, grid, dim3(256), 0, "lightning_step_kernel", l);
    if (l.dim <= 128) return md_launch_ex(ctx, lightning_step_kernel<T, 16>, grid, dim3(256), 0, "lightning_step_kernel", l);
    return md_launch_ex(ctx, lightning_step_kernel<T, 32>, grid, dim3(256), 0, "lightning_step_kernel", l);
}

constexpr int C = 64;   // tokens per chunk

// DP / VP: dim and vdim rounded up to 16, NW = DP / 16 warps own 16 state rows each in the update; the outputs' 64 rows are
// dealt to 4 row groups x NH column halves.
template <int DP, int VP>
struct ChunkShape {
    static constexpr int WARPS = DP / 16 < 4 ? 4 : DP / 16;       // 4 or 8
    static constexpr int UW = DP / 16;                             // warps with state rows
    static constexpr int NH = WARPS / 4;                           // column halves of the outputs
    static constexpr int PQ = DP + 8, PV = VP + 8;
    static constexpr size_t SMEM = (size_t)(2 * C * PQ + 3 * C * PV + 2 * DP * PV) * 2 + (C + 4 + C * NH) * 4;
};

template <int DP, int VP, bool OUT>
__global__ void __launch_bounds__((ChunkShape<DP, VP>::WARPS * 32))
lightning_chunk_kernel(const __grid_constant__ md_lightning p, float* seg_state, int chunks_per_seg, int n_seg) {
    using namespace mb;
    using Sh = ChunkShape<DP, VP>;
    constexpr int PQ = Sh::PQ, PV = Sh::PV, THREADS = Sh::WARPS * 32, NV = VP / 8;
    extern __shared__ __align__(16) unsigned char sm[];
    __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(sm);     // [64][PQ]
    __nv_bfloat16* Ks = Qs + C * PQ;
    __nv_bfloat16* Vs = Ks + C * PQ;                               // [64][PV] values, then decayed values as hi and lo
    __nv_bfloat16* Vh = Vs + C * PV;
    __nv_bfloat16* Vl = Vh + C * PV;
    __nv_bfloat16* Sh_hi = Vl + C * PV;                            // [DP][PV] state as hi and lo
    __nv_bfloat16* Sh_lo = Sh_hi + DP * PV;
    float* pw = reinterpret_cast<float*>(Sh_lo + DP * PV);         // lambda^0 .. lambda^64
    float* rowsq = pw + C + 4;                                     // [NH][64]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int seg = blockIdx.x, h = blockIdx.y, dim = p.dim, vdim = p.vdim;
    const float lambda = p.decay[h];
    if (tid <= C) pw[tid] = powf(lambda, (float)tid);
    md_pdl_launch_dependents();
    md_pdl_wait();
    const __nv_bfloat16* base = reinterpret_cast<const __nv_bfloat16*>(p.qkvg);
    const int Qc = h * dim, Kc = p.heads * dim + h * dim, Vc = 2 * p.heads * dim + h * vdim, Gc = Vc + p.heads * vdim;

    // state accumulators: rows warp * 16 + g (+ 8), columns nt * 8 + 2 t (+ 1)
    float S[NV][4];
    const bool updates = warp < Sh::UW;
    float* st = n_seg > 1 ? seg_state + ((size_t)seg * p.heads + h) * dim * vdim : p.state[0] + (size_t)h * dim * vdim;
#pragma unroll
    for (int nt = 0; nt < NV; ++nt) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int d = warp * 16 + g + (e >> 1) * 8, v = nt * 8 + 2 * t + (e & 1);
            S[nt][e] = OUT && updates && d < dim && v < vdim ? st[(size_t)d * vdim + v] : 0.f;
        }
    }
    const int total = (p.rows + C - 1) / C, c_end = min(total, (seg + 1) * chunks_per_seg);
    for (int chunk = seg * chunks_per_seg; chunk < c_end; ++chunk) {
        const int t0 = chunk * C, len = min(C, p.rows - t0);
        __syncthreads();    // the previous chunk's readers of shared memory are done (and pw is there)
        for (int i = tid; i < C * (DP / 8); i += THREADS) {
            const int r = i / (DP / 8), c = (i % (DP / 8)) * 8;
            const bool in = r < len && c < dim;
            const __nv_bfloat16* row = base + (size_t)(t0 + r) * p.row_stride;
            if (OUT) {
                if (in) cp_async16(smem_u32(Qs + r * PQ + c), row + Qc + c);
                else *reinterpret_cast<uint4*>(Qs + r * PQ + c) = make_uint4(0, 0, 0, 0);
            }
            if (in) cp_async16(smem_u32(Ks + r * PQ + c), row + Kc + c);
            else *reinterpret_cast<uint4*>(Ks + r * PQ + c) = make_uint4(0, 0, 0, 0);
        }
        cp_async_commit();
        for (int i = tid; i < C * (VP / 8); i += THREADS) {
            const int r = i / (VP / 8), c = (i % (VP / 8)) * 8;
            uint4 u = make_uint4(0, 0, 0, 0);
            if (r < len && c < vdim) u = *reinterpret_cast<const uint4*>(base + (size_t)(t0 + r) * p.row_stride + Vc + c);
            if (OUT) *reinterpret_cast<uint4*>(Vs + r * PV + c) = u;
            const float w = r < len ? pw[len - 1 - r] : 0.f;
            const uint32_t x[4] = {u.x, u.y, u.z, u.w};
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int j = 0; j < 4; ++j)
                split2(__uint_as_float(x[j] << 16) * w, __uint_as_float(x[j] & 0xffff0000u) * w, hi[j], lo[j]);
            *reinterpret_cast<uint4*>(Vh + r * PV + c) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
            *reinterpret_cast<uint4*>(Vl + r * PV + c) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
        }
        if (OUT && updates) {   // the state this chunk starts from
#pragma unroll
            for (int nt = 0; nt < NV; ++nt) {
#pragma unroll
                for (int rr = 0; rr < 2; ++rr) {
                    const int at = (warp * 16 + g + rr * 8) * PV + nt * 8 + 2 * t;
                    uint32_t hi, lo;
                    split2(S[nt][2 * rr], S[nt][2 * rr + 1], hi, lo);
                    *reinterpret_cast<uint32_t*>(Sh_hi + at) = hi;
                    *reinterpret_cast<uint32_t*>(Sh_lo + at) = lo;
                }
            }
        }
        cp_async_wait<0>();
        __syncthreads();
        if (OUT) {
            const int rg = warp & 3, nh = warp >> 2;
            constexpr int NB = VP / 16 / Sh::NH;      // 16-column blocks of this warp
            float o[2 * NB][4];
#pragma unroll
            for (int i = 0; i < 2 * NB; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
            float s[C / 8][4];
#pragma unroll
            for (int i = 0; i < C / 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
#pragma unroll
            for (int ks = 0; ks < DP / 16; ++ks) {
                uint32_t q[4];
                ldsm_x4(smem_u32(Qs + (rg * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PQ + ks * 16 + (lane >> 4) * 8), q);
#pragma unroll
                for (int np = 0; np < C / 16; ++np) {
                    if (np <= rg) {     // keys after the row group's last query see zero weights
                        uint32_t b[4];
                        ldsm_x4(smem_u32(Ks + (np * 16 + (lane & 7) + (lane >> 4) * 8) * PQ + ks * 16 + ((lane >> 3) & 1) * 8), b);
                        mma(s[2 * np], q[0], q[1], q[2], q[3], b[0], b[1]);
                        mma(s[2 * np + 1], q[0], q[1], q[2], q[3], b[2], b[3]);
                    }
                }
#pragma unroll
                for (int nb = 0; nb < NB; ++nb) {
                    const int at = (ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PV + (nh * NB + nb) * 16 + (lane >> 4) * 8;
                    uint32_t b[4];
                    ldsm_x4_t(smem_u32(Sh_hi + at), b);
                    mma(o[2 * nb], q[0], q[1], q[2], q[3], b[0], b[1]);
                    mma(o[2 * nb + 1], q[0], q[1], q[2], q[3], b[2], b[3]);
                    ldsm_x4_t(smem_u32(Sh_lo + at), b);
                    mma(o[2 * nb], q[0], q[1], q[2], q[3], b[0], b[1]);
                    mma(o[2 * nb + 1], q[0], q[1], q[2], q[3], b[2], b[3]);
                }
            }
            const int i0 = rg * 16 + g;      // rows i0 and i0 + 8 of the chunk
            const float f0 = pw[i0 + 1], f1 = pw[i0 + 9];
#pragma unroll
            for (int i = 0; i < 2 * NB; ++i) {
                o[i][0] *= f0; o[i][1] *= f0;
                o[i][2] *= f1; o[i][3] *= f1;
            }
#pragma unroll
            for (int nt = 0; nt < C / 8; ++nt) {
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int d = i0 + (e >> 1) * 8 - (nt * 8 + 2 * t + (e & 1));
                    s[nt][e] = d >= 0 ? s[nt][e] * pw[d >= 0 ? d : 0] : 0.f;
                }
            }
#pragma unroll
            for (int kk = 0; kk < C / 16; ++kk) {
                if (kk > rg) break;
                uint32_t hi[4], lo[4];
                split2(s[2 * kk][0], s[2 * kk][1], hi[0], lo[0]);
                split2(s[2 * kk][2], s[2 * kk][3], hi[1], lo[1]);
                split2(s[2 * kk + 1][0], s[2 * kk + 1][1], hi[2], lo[2]);
                split2(s[2 * kk + 1][2], s[2 * kk + 1][3], hi[3], lo[3]);
#pragma unroll
                for (int nb = 0; nb < NB; ++nb) {
                    uint32_t b[4];
                    ldsm_x4_t(smem_u32(Vs + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PV + (nh * NB + nb) * 16 + (lane >> 4) * 8), b);
                    mma(o[2 * nb], hi[0], hi[1], hi[2], hi[3], b[0], b[1]);
                    mma(o[2 * nb + 1], hi[0], hi[1], hi[2], hi[3], b[2], b[3]);
                    mma(o[2 * nb], lo[0], lo[1], lo[2], lo[3], b[0], b[1]);
                    mma(o[2 * nb + 1], lo[0], lo[1], lo[2], lo[3], b[2], b[3]);
                }
            }
#pragma unroll
            for (int rr = 0; rr < 2; ++rr) {
                const int i = i0 + rr * 8;
                const size_t row = (size_t)t0 + i;
                float sq = 0.f;
#pragma unroll
                for (int nt = 0; nt < 2 * NB; ++nt) {
                    const int v = nh * NB * 16 + nt * 8 + 2 * t;
                    const float x = o[nt][2 * rr], y = o[nt][2 * rr + 1];
                    sq = fmaf(x, x, fmaf(y, y, sq));     // columns past vdim are zero
                    if (i < len && v < vdim) {
                        const uint32_t gt = *reinterpret_cast<const uint32_t*>(base + row * p.row_stride + Gc + v);
                        const float2 nw = *reinterpret_cast<const float2*>(p.norm_w + h * vdim + v);
                        *reinterpret_cast<uint32_t*>(reinterpret_cast<__nv_bfloat16*>(p.out) + row * (p.heads * vdim) + h * vdim + v) =
                            md_pack_bf16(x * nw.x * __uint_as_float(gt << 16), y * nw.y * __uint_as_float(gt & 0xffff0000u));
                    }
                }
                sq += __shfl_xor_sync(0xffffffffu, sq, 1);
                sq += __shfl_xor_sync(0xffffffffu, sq, 2);
                if (t == 0) rowsq[nh * C + i] = sq;
            }
            __syncthreads();
            const int parts = p.ssq_parts / p.heads;     // the head's sum goes to its first entry
            for (int i = tid; i < len * parts; i += THREADS) {
                const int r = i / parts, k = i % parts;
                float v = 0.f;
                if (k == 0)
                    for (int n = 0; n < Sh::NH; ++n) v += rowsq[n * C + r];
                p.ssq[(size_t)(t0 + r) * p.ssq_parts + h * parts + k] = v;
            }
        }
        if (updates && (!OUT || seg == n_seg - 1 || chunk + 1 < c_end)) {
            const float f = pw[len];
#pragma unroll
            for (int nt = 0; nt < NV; ++nt) {
#pragma unroll
                for (int e = 0; e < 4; ++e) S[nt][e] *= f;
            }
#pragma unroll
            for (int kk = 0; kk < C / 16; ++kk) {
                uint32_t a[4];
                ldsm_x4_t(smem_u32(Ks + (kk * 16 + (lane & 7) + (lane >> 4) * 8) * PQ + warp * 16 + ((lane >> 3) & 1) * 8), a);
#pragma unroll
                for (int nb = 0; nb < VP / 16; ++nb) {
                    const int at = (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PV + nb * 16 + (lane >> 4) * 8;
                    uint32_t b[4];
                    ldsm_x4_t(smem_u32(Vh + at), b);
                    mma(S[2 * nb], a[0], a[1], a[2], a[3], b[0], b[1]);
                    mma(S[2 * nb + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
                    ldsm_x4_t(smem_u32(Vl + at), b);
                    mma(S[2 * nb], a[0], a[1], a[2], a[3], b[0], b[1]);
                    mma(S[2 * nb + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
                }
            }
        }
    }
    if (!updates || (OUT && seg != n_seg - 1)) return;
    float* dst = OUT ? p.state[0] + (size_t)h * dim * vdim : st;
#pragma unroll
    for (int nt = 0; nt < NV; ++nt) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int d = warp * 16 + g + (e >> 1) * 8, v = nt * 8 + 2 * t + (e & 1);
            if (d < dim && v < vdim) dst[(size_t)d * vdim + v] = S[nt][e];
        }
    }
}

// In: entry s of seg_state = what segment s adds to a zero state (s < n_seg - 1).  Out: the state segment s starts from.
__global__ void __launch_bounds__(256)
lightning_carry_kernel(const __grid_constant__ md_lightning p, float* seg_state, int seg_tokens, int n_seg) {
    md_pdl_launch_dependents();
    md_pdl_wait();
    const size_t per = (size_t)p.dim * p.vdim, n = p.heads * per;
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    const float f = powf(p.decay[i / per], (float)seg_tokens);
    float S = p.state[0][i];
    for (int s0 = 0; s0 < n_seg; s0 += 16) {     // sixteen contributions requested at a time
        float u[16];
#pragma unroll
        for (int k = 0; k < 16; ++k) u[k] = s0 + k < n_seg - 1 ? seg_state[(s0 + k) * n + i] : 0.f;
#pragma unroll
        for (int k = 0; k < 16; ++k) {
            if (s0 + k < n_seg) seg_state[(s0 + k) * n + i] = S;
            S = fmaf(f, S, u[k]);
        }
    }
}

template <int DP, int VP>
int launch_chunks_as(md_ctx* ctx, const md_lightning& l) {
    using Sh = ChunkShape<DP, VP>;
    auto out = lightning_chunk_kernel<DP, VP, true>;
    auto acc = lightning_chunk_kernel<DP, VP, false>;
    if (Sh::SMEM > 48 * 1024) {
        MD_CUDA(ctx, cudaFuncSetAttribute(out, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)Sh::SMEM));
        MD_CUDA(ctx, cudaFuncSetAttribute(acc, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)Sh::SMEM));
    }
    // segments: about three blocks per SM; two chunks are not worth the two further kernels
    const int chunks = (l.rows + C - 1) / C;
    int n_seg = (3 * ctx->sm_count + l.heads - 1) / l.heads;
    if (n_seg > chunks) n_seg = chunks;
    if (chunks <= 2) n_seg = 1;
    const int per = (chunks + n_seg - 1) / n_seg;
    n_seg = (chunks + per - 1) / per;
    const size_t n = (size_t)l.heads * l.dim * l.vdim;
    float* seg_state = nullptr;
    if (n_seg > 1) {
        void* scratch = nullptr;
        MD_TRY(md_scratch(ctx, n_seg * n * sizeof(float), &scratch));
        seg_state = reinterpret_cast<float*>(scratch);
        MD_TRY(md_launch_ex(ctx, acc, dim3((unsigned)(n_seg - 1), (unsigned)l.heads), dim3(Sh::WARPS * 32), Sh::SMEM,
                            "lightning_chunk_kernel", l, seg_state, per, n_seg));
        MD_TRY(md_launch_ex(ctx, lightning_carry_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, "lightning_carry_kernel", l,
                            seg_state, per * C, n_seg));
    }
    return md_launch_ex(ctx, out, dim3((unsigned)n_seg, (unsigned)l.heads), dim3(Sh::WARPS * 32), Sh::SMEM, "lightning_chunk_kernel", l,
                        seg_state, per, n_seg);
}

// rounded up to the instantiated sizes; what is past dim or vdim is zero in shared memory
int launch_chunks(md_ctx* ctx, const md_lightning& l) {
    const bool d64 = l.dim <= 64, v64 = l.vdim <= 64;
    if (d64) return v64 ? launch_chunks_as<64, 64>(ctx, l) : launch_chunks_as<64, 128>(ctx, l);
    return v64 ? launch_chunks_as<128, 64>(ctx, l) : launch_chunks_as<128, 128>(ctx, l);
}
bool chunks_ok(const md_lightning& l) {
    return l.seqs == 1 && (l.dim % 8) == 0 && (l.vdim % 8) == 0 && l.dim <= 128 && l.vdim <= 128 && (l.row_stride % 8) == 0 &&
           ((reinterpret_cast<uintptr_t>(l.qkvg) | reinterpret_cast<uintptr_t>(l.out)) & 15) == 0;
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
    if (l.rows == 1 && l.dim <= 256 && decode)
        return dtype == MD_DTYPE_F32 ? launch_step<float>(ctx, l) : launch_step<__nv_bfloat16>(ctx, l);
    if (dtype == MD_DTYPE_BF16 && chunks_ok(l)) return launch_chunks(ctx, l);
    return dtype == MD_DTYPE_F32 ? launch_scan<float>(ctx, l) : launch_scan<__nv_bfloat16>(ctx, l);
}
