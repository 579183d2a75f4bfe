// Grouped-query attention with a logarithmic distance bias, a sliding window with kept first tokens, values that are the
// keys, and one output gate per head (md_win_attn in stack.cuh).
//   append_keys_kernel      new key rows into the cache [kv_heads][max_seq][dim]
//   window_attention_kernel any element type and head size: one warp per (query, head), lanes over the head's dims
//   window_prefill_kernel   bfloat16 prompts: 64 queries x 64 keys per step on tensor cores.  One tile in shared memory is
//                           both the keys and the values.  The distance bias depends on i - j alone, so a step computes the
//                           127 values its tile can need once (one logarithm per thread) and masks through the same table
//                           (infinite bias outside the window).  Tiles are the window's, preceded by those of the kept
//                           first tokens.  Weights enter the second product as two bfloat16 terms (mma_bf16.cuh).
//   window_decode_kernel    bfloat16, one new token per sequence: a block takes 64 of the visible keys of one key head for
//                           all query heads that share it (each key is read once), appends the new key, and the last
//                           block of a key head merges the partial sums.
#include "mma_bf16.cuh"

#include <algorithm>

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

constexpr float LOG2E = 1.4426950408889634f;
constexpr int BQ = 64, BK = 64;

// 2^x by the hardware instruction (relative error about 2^-22), without exp2f's care for denormal results
__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// keys (8 values per thread) into the cache
__global__ void __launch_bounds__(256)
append_keys_vec_kernel(const __grid_constant__ md_win_attn p) {
    md_pdl_launch_dependents();
    md_pdl_wait();
    const int per = p.kv_heads * p.dim / 8;
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long long)p.rows * per) return;
    const int t = (int)(i / per), c = (int)(i % per) * 8, g = c / p.dim, d = c % p.dim;
    const __nv_bfloat16* src = reinterpret_cast<const __nv_bfloat16*>(p.qkg) + (size_t)t * p.row_stride + p.heads * p.dim + c;
    *reinterpret_cast<uint4*>(reinterpret_cast<__nv_bfloat16*>(p.kc[0]) + ((size_t)g * p.max_seq + p.pos0 + t) * p.dim + d) =
        *reinterpret_cast<const uint4*>(src);
}

// DP: head size rounded up to a multiple of 16 (the pad is zero in shared memory)
template <int DP>
__global__ void __launch_bounds__(128, DP <= 64 ? 4 : DP <= 96 ? 3 : DP <= 128 ? 2 : 1)
window_prefill_kernel(const __grid_constant__ md_win_attn p) {
    using namespace mb;
    constexpr int PITCH = DP + 8, CH = DP / 8;
    constexpr bool Q_REGS = DP <= 128;    // longer heads re-read their query fragments from shared memory
    extern __shared__ __align__(16) unsigned char sm[];
    __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(sm);
    __nv_bfloat16* Ks = Qs + BQ * PITCH;                     // two tiles
    float* tab = reinterpret_cast<float*>(Ks + 2 * BK * PITCH);   // two tables of 128: bias of distance index - 63
    md_pdl_launch_dependents();
    md_pdl_wait();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int q0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * BQ, h = blockIdx.y, kvh = h / (p.heads / p.kv_heads);
    const __nv_bfloat16* qb = reinterpret_cast<const __nv_bfloat16*>(p.qkg) + h * p.dim;
    const __nv_bfloat16* kb = reinterpret_cast<const __nv_bfloat16*>(p.kc[0]) + (size_t)kvh * p.max_seq * p.dim;
    const int rows = min(BQ, p.rows - q0), real = p.dim / 8;
    const float r1 = p.r1[h] * LOG2E, r2 = p.r2[h], scale = p.scale * LOG2E;
    const int window = p.window > 0 ? p.window : 0x3fffffff;

    for (int i = tid; i < BQ * CH; i += 128) {
        const int r = i / CH, c = i % CH;
        if (r < rows && c < real) cp_async16(smem_u32(Qs + r * PITCH + c * 8), qb + (size_t)(q0 + r) * p.row_stride + c * 8);
        else *reinterpret_cast<uint4*>(Qs + r * PITCH + c * 8) = make_uint4(0, 0, 0, 0);
    }
    // positions: query row r is at P0 + r; the keys of the window of the block start at `first`
    const int P0 = p.pos0 + q0, last = P0 + rows - 1;
    const int start = max(0, P0 - window + 1) / BK * BK;                    // first tile of the windows
    const int kept = (min(p.keep_first, start) + BK - 1) / BK;              // tiles of kept tokens ahead of it
    const int n_tiles = kept + (last - start) / BK + 1;
    auto tile_key = [&](int i) { return i < kept ? i * BK : start + (i - kept) * BK; };
    auto load_tile = [&](int i) {
        const int k0 = tile_key(i), buf = i & 1;
        for (int j = tid; j < BK * CH; j += 128) {
            const int r = j / CH, c = j % CH;
            __nv_bfloat16* dst = Ks + (size_t)(buf * BK + r) * PITCH + c * 8;
            if (k0 + r <= last && c < real) cp_async16(smem_u32(dst), kb + (size_t)(k0 + r) * p.dim + c * 8);
            else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
        cp_async_commit();
        const int d = P0 - k0 + tid - (BK - 1);   // distance this thread's entry stands for
        const bool by_key = k0 < p.keep_first;    // a tile with kept tokens masks per element
        tab[buf * 128 + tid] = d < 0 || (!by_key && d >= window) ? INFINITY : r1 * log1pf(r2 * (float)d);
    };
    load_tile(0);
    uint32_t qf[Q_REGS ? DP / 16 : 1][4];
    float o[DP / 8][4];
#pragma unroll
    for (int i = 0; i < DP / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
    const int q_row = warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, q_col = (lane >> 4) * 8;

    for (int it = 0; it < n_tiles; ++it) {
        const int k0 = tile_key(it), buf = it & 1;
        cp_async_wait<0>();
        __syncthreads();                              // tile `it` is there, and nobody reads the other buffer any more
        if (it + 1 < n_tiles) load_tile(it + 1);      // in flight while this tile is worked on
        if (Q_REGS && it == 0) {
#pragma unroll
            for (int ks = 0; ks < DP / 16; ++ks) ldsm_x4(smem_u32(Qs + q_row * PITCH + ks * 16 + q_col), qf[Q_REGS ? ks : 0]);
        }
        const __nv_bfloat16* K = Ks + (size_t)buf * BK * PITCH;
        float s[BK / 8][4];
#pragma unroll
        for (int i = 0; i < BK / 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
#pragma unroll
        for (int ks = 0; ks < DP / 16; ++ks) {
            if (!Q_REGS) ldsm_x4(smem_u32(Qs + q_row * PITCH + ks * 16 + q_col), qf[0]);
            const uint32_t (&q)[4] = qf[Q_REGS ? ks : 0];
#pragma unroll
            for (int np = 0; np < BK / 16; ++np) {
                uint32_t b[4];
                ldsm_x4(smem_u32(K + (np * 16 + (lane & 7) + (lane >> 4) * 8) * PITCH + ks * 16 + ((lane >> 3) & 1) * 8), b);
                mma(s[2 * np], q[0], q[1], q[2], q[3], b[0], b[1]);
                mma(s[2 * np + 1], q[0], q[1], q[2], q[3], b[2], b[3]);
            }
        }
        const bool by_key = k0 < p.keep_first;
        const float* tb = tab + buf * 128 + (BK - 1) + warp * 16 + g - 2 * t;
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int nt = 0; nt < BK / 8; ++nt) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int rr = e >> 1, col = nt * 8 + (e & 1);     // key k0 + col + 2 t, query row warp * 16 + g + 8 rr
                float v = fmaf(s[nt][e], scale, -tb[rr * 8 - col]);
                if (by_key) {
                    const int key = k0 + col + 2 * t, d = P0 + warp * 16 + g + rr * 8 - key;
                    if (d >= window && key >= p.keep_first) v = -INFINITY;
                }
                s[nt][e] = v;
                mx[rr] = fmaxf(mx[rr], v);
            }
        }
        float corr[2], m_use[2], rs[2] = {0.f, 0.f};
#pragma unroll
        for (int rr = 0; rr < 2; ++rr) {
            mx[rr] = fmaxf(mx[rr], __shfl_xor_sync(0xffffffffu, mx[rr], 1));
            mx[rr] = fmaxf(mx[rr], __shfl_xor_sync(0xffffffffu, mx[rr], 2));
            const float mn = fmaxf(m_run[rr], mx[rr]);
            m_use[rr] = mn == -INFINITY ? 0.f : mn;
            corr[rr] = m_run[rr] == -INFINITY ? 0.f : ex2(m_run[rr] - m_use[rr]);
            m_run[rr] = mn;
        }
#pragma unroll
        for (int nt = 0; nt < BK / 8; ++nt) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                s[nt][e] = ex2(s[nt][e] - m_use[e >> 1]);
                rs[e >> 1] += s[nt][e];
            }
        }
#pragma unroll
        for (int rr = 0; rr < 2; ++rr) {
            rs[rr] += __shfl_xor_sync(0xffffffffu, rs[rr], 1);
            rs[rr] += __shfl_xor_sync(0xffffffffu, rs[rr], 2);
            l_run[rr] = l_run[rr] * corr[rr] + rs[rr];
        }
        if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {   // a maximum of this warp's rows moved
#pragma unroll
            for (int i = 0; i < DP / 8; ++i) {
                o[i][0] *= corr[0]; o[i][1] *= corr[0];
                o[i][2] *= corr[1]; o[i][3] *= corr[1];
            }
        }
#pragma unroll
        for (int kk = 0; kk < BK / 16; ++kk) {
            uint32_t hi[4], lo[4];
            split2(s[2 * kk][0], s[2 * kk][1], hi[0], lo[0]);
            split2(s[2 * kk][2], s[2 * kk][3], hi[1], lo[1]);
            split2(s[2 * kk + 1][0], s[2 * kk + 1][1], hi[2], lo[2]);
            split2(s[2 * kk + 1][2], s[2 * kk + 1][3], hi[3], lo[3]);
#pragma unroll
            for (int dp = 0; dp < DP / 16; ++dp) {
                uint32_t b[4];
                ldsm_x4_t(smem_u32(K + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PITCH + dp * 16 + (lane >> 4) * 8), b);
                mma(o[2 * dp], hi[0], hi[1], hi[2], hi[3], b[0], b[1]);
                mma(o[2 * dp + 1], hi[0], hi[1], hi[2], hi[3], b[2], b[3]);
                mma(o[2 * dp], lo[0], lo[1], lo[2], lo[3], b[0], b[1]);
                mma(o[2 * dp + 1], lo[0], lo[1], lo[2], lo[3], b[2], b[3]);
            }
        }
    }
#pragma unroll
    for (int rr = 0; rr < 2; ++rr) {
        const int r = warp * 16 + g + rr * 8;
        if (r >= rows) continue;
        const __nv_bfloat16* row = reinterpret_cast<const __nv_bfloat16*>(p.qkg) + (size_t)(q0 + r) * p.row_stride;
        const float f = __bfloat162float(row[(p.heads + p.kv_heads) * p.dim + h]) / l_run[rr];
        __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + (size_t)(q0 + r) * p.heads * p.dim + h * p.dim;
#pragma unroll
        for (int nt = 0; nt < DP / 8; ++nt)
            if (nt < real) *reinterpret_cast<uint32_t*>(out + nt * 8 + 2 * t) = md_pack_bf16(o[nt][2 * rr] * f, o[nt][2 * rr + 1] * f);
    }
}

constexpr int DEC_KEYS = 64, DEC_THREADS = 128, DEC_MAX_DIM = 256, DEC_MAX_GROUP = DEC_THREADS;

// visible keys of a token at `pos`, in order: the kept ones ahead of the window, then the window's; `index` counts them
__device__ __forceinline__ int visible_key(int index, int kept, int first) { return index < kept ? index : first + (index - kept); }

__global__ void __launch_bounds__(DEC_THREADS)
window_decode_kernel(const __grid_constant__ md_win_attn p, float* partial, unsigned* tickets, int max_splits) {
    using namespace mb;
    extern __shared__ __align__(16) unsigned char sm[];
    const int dim = p.dim, dp = (dim + 15) & ~15, pitch = dp + 8, R = p.heads / p.kv_heads;
    __nv_bfloat16* Ks = reinterpret_cast<__nv_bfloat16*>(sm);        // [64][pitch]
    __nv_bfloat16* Qs = Ks + DEC_KEYS * pitch;                        // [8][pitch], eight heads at a time
    float* Ps = reinterpret_cast<float*>(Qs + 8 * pitch);             // [8][64]
    float* ms = Ps + 8 * DEC_KEYS;                                    // [4][8] maxima, then [4][8] sums
    __shared__ int last_s;
    __shared__ float gates[DEC_MAX_GROUP], rs1[DEC_MAX_GROUP], rs2[DEC_MAX_GROUP];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int split = blockIdx.x, kvh = blockIdx.y, seq = blockIdx.z;
    const int pos = *p.pos_dev[seq];   // written by the kernel that ended the previous step
    const int window = p.window > 0 ? p.window : 0x3fffffff;
    const int first = max(0, pos - window + 1), kept = min(p.keep_first, first), visible = kept + pos - first + 1;
    const int splits = (visible + DEC_KEYS - 1) / DEC_KEYS;
    md_pdl_launch_dependents();
    if (split >= splits) return;
    const int n = min(DEC_KEYS, visible - split * DEC_KEYS), ch = dp / 8, real = dim / 8;
    __nv_bfloat16* cache = reinterpret_cast<__nv_bfloat16*>(p.kc[seq]) + (size_t)kvh * p.max_seq * dim;
    const bool newest = split == splits - 1;                          // holds the new key as its last one
    // the cached keys were written by earlier steps: requested before the wait for this step's projections
    for (int i = tid; i < DEC_KEYS * ch; i += DEC_THREADS) {
        const int r = i / ch, c = i % ch;
        if (r < n - (newest ? 1 : 0) && c < real)
            cp_async16(smem_u32(Ks + r * pitch + c * 8), cache + (size_t)visible_key(split * DEC_KEYS + r, kept, first) * dim + c * 8);
        else if (!(newest && r == n - 1 && c < real))
            *reinterpret_cast<uint4*>(Ks + r * pitch + c * 8) = make_uint4(0, 0, 0, 0);
    }
    cp_async_commit();
    if (tid < R) {
        rs1[tid] = p.r1[kvh * R + tid];
        rs2[tid] = p.r2[kvh * R + tid];
    }
    md_pdl_wait();
    const __nv_bfloat16* row = reinterpret_cast<const __nv_bfloat16*>(p.qkg) + (size_t)seq * p.row_stride;
    if (newest && tid < real) {
        const uint4 k = __ldcg(reinterpret_cast<const uint4*>(row + (p.heads + kvh) * dim + tid * 8));
        *reinterpret_cast<uint4*>(Ks + (n - 1) * pitch + tid * 8) = k;
        *reinterpret_cast<uint4*>(cache + (size_t)pos * dim + tid * 8) = k;
    }
    if (tid < R) gates[tid] = __bfloat162float(row[(p.heads + p.kv_heads) * dim + kvh * R + tid]);
    const size_t slot = (size_t)seq * p.kv_heads + kvh;
    float* mine = partial + (slot * max_splits + split) * R * (dim + 2);
    for (int h0 = 0; h0 < R; h0 += 8) {
        const int heads = min(8, R - h0);
        for (int i = tid; i < 8 * ch; i += DEC_THREADS) {
            const int r = i / ch, c = i % ch;
            *reinterpret_cast<uint4*>(Qs + r * pitch + c * 8) =
                r < heads && c < real ? __ldcg(reinterpret_cast<const uint4*>(row + (kvh * R + h0 + r) * dim + c * 8)) : make_uint4(0, 0, 0, 0);
        }
        if (h0 == 0) cp_async_wait<0>();
        __syncthreads();
        // S^T: 16 keys per warp x 8 heads
        float s[4] = {0.f, 0.f, 0.f, 0.f};
        for (int ks = 0; ks < dp / 16; ++ks) {
            uint32_t a[4];
            ldsm_x4(smem_u32(Ks + (warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * pitch + ks * 16 + (lane >> 4) * 8), a);
            const uint32_t b0 = *reinterpret_cast<const uint32_t*>(Qs + g * pitch + ks * 16 + 2 * t);
            const uint32_t b1 = *reinterpret_cast<const uint32_t*>(Qs + g * pitch + ks * 16 + 2 * t + 8);
            mma(s, a[0], a[1], a[2], a[3], b0, b1);
        }
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int e = 0; e < 4; ++e) {      // key g + 8 (e >> 1), head 2 t + (e & 1)
            const int r = warp * 16 + g + (e >> 1) * 8, hh = 2 * t + (e & 1);
            float v = -INFINITY;
            if (r < n && hh < heads) {
                const int h = h0 + hh, d = pos - visible_key(split * DEC_KEYS + r, kept, first);
                v = (s[e] * p.scale - rs1[h] * log1pf(rs2[h] * (float)d)) * LOG2E;
            }
            s[e] = v;
            mx[e & 1] = fmaxf(mx[e & 1], v);
        }
#pragma unroll
        for (int o = 4; o < 32; o <<= 1) {
            mx[0] = fmaxf(mx[0], __shfl_xor_sync(0xffffffffu, mx[0], o));
            mx[1] = fmaxf(mx[1], __shfl_xor_sync(0xffffffffu, mx[1], o));
        }
        if (g == 0) {
            ms[warp * 8 + 2 * t] = mx[0];
            ms[warp * 8 + 2 * t + 1] = mx[1];
        }
        __syncthreads();
        float sum[2] = {0.f, 0.f};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int hh = 2 * t + (e & 1), r = warp * 16 + g + (e >> 1) * 8;
            const float m = fmaxf(fmaxf(ms[hh], ms[8 + hh]), fmaxf(ms[16 + hh], ms[24 + hh]));
            const float w = s[e] == -INFINITY ? 0.f : exp2f(s[e] - m);
            Ps[hh * DEC_KEYS + r] = w;
            sum[e & 1] += w;
        }
#pragma unroll
        for (int o = 4; o < 32; o <<= 1) {
            sum[0] += __shfl_xor_sync(0xffffffffu, sum[0], o);
            sum[1] += __shfl_xor_sync(0xffffffffu, sum[1], o);
        }
        if (g == 0) {
            ms[32 + warp * 8 + 2 * t] = sum[0];
            ms[32 + warp * 8 + 2 * t + 1] = sum[1];
        }
        __syncthreads();
        if (tid < heads) {
            mine[(h0 + tid) * (dim + 2)] = fmaxf(fmaxf(ms[tid], ms[8 + tid]), fmaxf(ms[16 + tid], ms[24 + tid]));
            mine[(h0 + tid) * (dim + 2) + 1] = ms[32 + tid] + ms[40 + tid] + ms[48 + tid] + ms[56 + tid];
        }
        // O^T: 16 dims per turn and warp x 8 heads, over the 64 keys
        for (int dt = warp; dt < dp / 16; dt += 4) {
            float o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int kk = 0; kk < DEC_KEYS / 16; ++kk) {
                uint32_t a[4], hi0, lo0, hi1, lo1;
                // rows of A are dims: matrices (dims 0-7, keys 0-7), (dims 8-15, keys 0-7), (dims 0-7, keys 8-15), ...
                ldsm_x4_t(smem_u32(Ks + (kk * 16 + (lane & 7) + (lane >> 4) * 8) * pitch + dt * 16 + ((lane >> 3) & 1) * 8), a);
                const float* pr = Ps + g * DEC_KEYS + kk * 16 + 2 * t;
                split2(pr[0], pr[1], hi0, lo0);
                split2(pr[8], pr[9], hi1, lo1);
                mma(o, a[0], a[1], a[2], a[3], hi0, hi1);
                mma(o, a[0], a[1], a[2], a[3], lo0, lo1);
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int d = dt * 16 + g + (e >> 1) * 8, hh = 2 * t + (e & 1);
                if (d < dim && hh < heads) mine[(h0 + hh) * (dim + 2) + 2 + d] = o[e];
            }
        }
        __syncthreads();
    }
    __threadfence();
    __syncthreads();
    if (splits > 1) {
        if (tid == 0) last_s = atomicAdd(tickets + slot, 1u) == (unsigned)splits - 1;
        __syncthreads();
        if (!last_s) return;
        __threadfence();
        if (tid == 0) tickets[slot] = 0u;
    }
    const float* base = partial + slot * max_splits * R * (dim + 2);
    const size_t step = (size_t)R * (dim + 2);
    for (int i = tid; i < R * dim; i += DEC_THREADS) {
        const int hh = i / dim, d = i % dim, h = kvh * R + hh;
        const float* b = base + (size_t)hh * (dim + 2);
        float m = -INFINITY, l = 0.f, o = 0.f;
        for (int s0 = 0; s0 < splits; s0 += 8) {       // eight partials requested at a time
            float pm[8], pl[8], po[8];
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                const bool live = s0 + u < splits;
                pm[u] = live ? __ldcg(b + (s0 + u) * step) : -INFINITY;
                pl[u] = live ? __ldcg(b + (s0 + u) * step + 1) : 0.f;
                po[u] = live ? __ldcg(b + (s0 + u) * step + 2 + d) : 0.f;
            }
            float mn = m;
#pragma unroll
            for (int u = 0; u < 8; ++u) mn = fmaxf(mn, pm[u]);
            const float c = m == -INFINITY ? 0.f : exp2f(m - mn);
            l *= c;
            o *= c;
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                const float f = pm[u] == -INFINITY ? 0.f : exp2f(pm[u] - mn);
                l = fmaf(pl[u], f, l);
                o = fmaf(po[u], f, o);
            }
            m = mn;
        }
        reinterpret_cast<__nv_bfloat16*>(p.out)[(size_t)seq * p.heads * dim + h * dim + d] = __float2bfloat16_rn(o / l * gates[hh]);
    }
}

bool vector_ok(const md_win_attn& a) {
    return (a.dim % 8) == 0 && a.dim <= DEC_MAX_DIM && (a.row_stride % 8) == 0 &&
           ((reinterpret_cast<uintptr_t>(a.qkg) | reinterpret_cast<uintptr_t>(a.out)) & 15) == 0;
}

template <int DP>
int launch_prefill_as(md_ctx* ctx, const md_win_attn& a) {
    constexpr size_t smem = (size_t)(BQ + 2 * BK) * (DP + 8) * 2 + 256 * sizeof(float);
    auto kern = window_prefill_kernel<DP>;
    if (smem > 48 * 1024) MD_CUDA(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    return md_launch_ex(ctx, kern, dim3((unsigned)((a.rows + BQ - 1) / BQ), (unsigned)a.heads), dim3(128), smem, "window_prefill_kernel", a);
}

int launch_prefill(md_ctx* ctx, const md_win_attn& a) {
    const long long n = (long long)a.rows * a.kv_heads * a.dim / 8;
    MD_TRY(md_launch_ex(ctx, append_keys_vec_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, "append_keys_kernel", a));
    if (a.dim <= 32) return launch_prefill_as<32>(ctx, a);
    if (a.dim <= 48) return launch_prefill_as<48>(ctx, a);
    if (a.dim <= 64) return launch_prefill_as<64>(ctx, a);
    if (a.dim <= 80) return launch_prefill_as<80>(ctx, a);
    if (a.dim <= 96) return launch_prefill_as<96>(ctx, a);
    if (a.dim <= 128) return launch_prefill_as<128>(ctx, a);
    if (a.dim <= 192) return launch_prefill_as<192>(ctx, a);
    return launch_prefill_as<256>(ctx, a);
}

int launch_decode(md_ctx* ctx, const md_win_attn& a) {
    const int R = a.heads / a.kv_heads, dp = (a.dim + 15) & ~15;
    // most keys a token can see: the kept ones and a window, or everything the cache holds
    const size_t most = a.window > 0 ? std::min<size_t>(a.max_seq, (size_t)a.window + a.keep_first) : a.max_seq;
    const int max_splits = (int)((most + DEC_KEYS - 1) / DEC_KEYS);
    if ((size_t)a.seqs * a.kv_heads > MD_COUNTER_WORDS)
        return md_fail(ctx, MD_ERR_UNSUPPORTED, "window attention: %d sequences of %d key heads exceed the arrival counters", a.seqs, a.kv_heads);
    void* scratch = nullptr;
    MD_TRY(md_scratch(ctx, (size_t)a.seqs * a.kv_heads * max_splits * R * (a.dim + 2) * sizeof(float), &scratch));
    const size_t smem = (size_t)(DEC_KEYS + 8) * (dp + 8) * 2 + (8 * DEC_KEYS + 64) * sizeof(float);
    return md_launch_ex(ctx, window_decode_kernel, dim3((unsigned)max_splits, (unsigned)a.kv_heads, (unsigned)a.seqs), dim3(DEC_THREADS),
                        smem, "window_decode_kernel", a, reinterpret_cast<float*>(scratch), ctx->counters, max_splits);
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
    if (dtype == MD_DTYPE_BF16 && vector_ok(a)) {
        if (decode && a.rows == 1 && a.heads / a.kv_heads <= DEC_MAX_GROUP) return launch_decode(ctx, a);
        if (!decode && a.seqs == 1) return launch_prefill(ctx, a);
    }
    if (a.dim > 32 * PER_LANE) return md_fail(ctx, MD_ERR_UNSUPPORTED, "window attention: head size %d > %d", a.dim, 32 * PER_LANE);
    return dtype == MD_DTYPE_F32 ? launch<float>(ctx, a) : launch<__nv_bfloat16>(ctx, a);
}
