// Mixture of experts (md_moe in stack.cuh): independent logistic scores, or a softmax over the chosen experts' logits, and
// an optional shared expert that every token takes, weighted with the logistic of the router's last row.
//
// Prompts (and every shape the kernels below cannot take):
//   moe_router_kernel, moe_router_mma_kernel
//                       scores and top choice per token (f32 sums of exact bfloat16 products, or f32 throughout), and each
//                       (token, expert) pair's rank within its expert
//   moe_permute_kernel  rows sorted by expert, every expert's rows starting at a multiple of 128
// then the two expert products run as grouped products over the sorted rows, and the weighted sum of a token's experts
// is taken where the residual is updated (md_glue::slot).  The shared expert's two products run over the tokens as they
// are, its rows land behind the sorted ones, and a token's last entry of slot and score points there.
//
// Up to eight bfloat16 tokens (a decode step), weights streamed as in gemv.cu:
//   moe_route_kernel    scores of all tokens; the last block to arrive chooses and lists the experts in use ("slots") with
//                       every token's weight in each (zero where the token does not use it)
//   moe_up_kernel       the slots' gated products, times the token's weight; the shared expert is one more slot
//   moe_down_kernel     one long product over all slots' columns, so the weighted sum needs no second pass
#include "mma_bf16.cuh"

namespace {

constexpr int MAX_EXPERTS = 512, MAX_TOP = 32;

// The `top` largest of the logits s[0 .. E) (shared memory, lowest index first among equals), by one warp:
// fn(k, expert, weight) in lane k.
template <class F>
__device__ __forceinline__ void warp_top(float* s, int E, int top, int kind, int lane, F&& fn) {
    float mine = -INFINITY, first = -INFINITY;
    int expert = 0;
    for (int k = 0; k < top; ++k) {
        float best = -INFINITY;
        int bi = 0;
        for (int e = lane; e < E; e += 32)
            if (s[e] > best) { best = s[e]; bi = e; }
#pragma unroll
        for (int o = 16; o; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (ob > best || (ob == best && oi < bi)) { best = ob; bi = oi; }
        }
        if (k == 0) first = best;
        if (lane == k) {
            mine = best;
            expert = bi;
        }
        if (lane == 0) s[bi] = -INFINITY;
        __syncwarp();
    }
    if (kind == MD_ROUTER_SOFTMAX) {
        mine = lane < top ? expf(mine - first) : 0.f;
        float sum = mine;
#pragma unroll
        for (int o = 16; o; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        mine /= sum;
    } else {
        mine = md_logistic(mine);
    }
    if (lane < top) fn(lane, expert, mine);
    __syncwarp();
}

// one warp per token
template <class T>
__global__ void __launch_bounds__(128)
moe_router_kernel(const T* __restrict__ h, const T* __restrict__ router, int rows, int W, int E, int shared, int top, int kind,
                  float* score, int* sel, int* rank, int* count) {
    __shared__ float s_all[4][MAX_EXPERTS + 1];
    md_pdl_launch_dependents();
    md_pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x * 4 + warp;
    if (t >= rows) return;
    float* s = s_all[warp];
    const T* hr = h + (size_t)t * W;
    for (int e = 0; e < E + shared; ++e) {
        const T* wr = router + (size_t)e * W;
        float z = 0.f;
        for (int c = lane; c < W; c += 32) z = fmaf(md_elem<T>::get(hr[c]), md_elem<T>::get(wr[c]), z);
#pragma unroll
        for (int o = 16; o; o >>= 1) z += __shfl_xor_sync(0xffffffffu, z, o);
        if (lane == 0) s[e] = z;
    }
    __syncwarp();
    if (shared && lane == 0) score[(size_t)t * (top + 1) + top] = md_logistic(s[E]);
    warp_top(s, E, top, kind, lane, [&](int k, int e, float v) {
        score[(size_t)t * (top + shared) + k] = v;
        sel[(size_t)t * top + k] = e;
        rank[(size_t)t * top + k] = atomicAdd(count + e, 1);
    });
}

template <class T>
__global__ void __launch_bounds__(256)
moe_permute_kernel(const T* __restrict__ h, int W, int E, int shared_row, int top, const int* __restrict__ sel,
                   const int* __restrict__ rank, const int* __restrict__ count, int* slot, int* tile_expert, int* n_blocks,
                   T* __restrict__ xs) {
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
    const int choices = top + (shared_row >= 0 ? 1 : 0);
    if (shared_row >= 0 && threadIdx.x == 0) slot[(size_t)t * choices + top] = shared_row + t;
    for (int k = 0; k < top; ++k) {
        const int e = sel[(size_t)t * top + k], row = first[e] * MD_GROUP_ROWS + rank[(size_t)t * top + k];
        if (threadIdx.x == 0) slot[(size_t)t * choices + k] = row;
        T* dst = xs + (size_t)row * W;
        if ((W * sizeof(T)) % 16 == 0) {
            for (int c = threadIdx.x; c < (int)(W * sizeof(T) / 16); c += blockDim.x)
                reinterpret_cast<uint4*>(dst)[c] = reinterpret_cast<const uint4*>(src)[c];
        } else if ((W % 4) == 0) {
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

__device__ __forceinline__ uint4 ldg_stream(const void* p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];"
                 : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w)
                 : "l"(p));
    return v;
}
__device__ __forceinline__ uint4 ld_act(const void* p) {
    uint4 v;
    asm volatile("ld.global.cg.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p) : "memory");
    return v;
}
// 32 k values of 16 rows (lo: rows g, hi: rows g + 8) against 8 columns: the order of k inside a sum is free, so a lane's
// 8 consecutive values feed two MMAs
__device__ __forceinline__ void mma_piece(float (&c)[4], const uint4& lo, const uint4& hi, const uint4& x) {
    mb::mma(c, lo.x, hi.x, lo.y, hi.y, x.x, x.y);
    mb::mma(c, lo.z, hi.z, lo.w, hi.w, x.z, x.w);
}

constexpr int RT = 16, RE = 64;   // tokens per block, experts per pass

constexpr int RW = 16;   // warps that split the width

__global__ void __launch_bounds__(RW * 32)
moe_router_mma_kernel(const __nv_bfloat16* h, const __nv_bfloat16* __restrict__ router, int rows, int W, int E, int shared, int top,
                      int kind, float* score, int* sel, int* rank, int* count) {
    const int EA = E + shared;   // rows of the router
    extern __shared__ float smf[];
    float (*part)[RT][RE] = reinterpret_cast<float (*)[RT][RE]>(smf);   // [RW]
    float* sc = smf + RW * RT * RE;                                      // [RT][EA]
    int* cnt = reinterpret_cast<int*>(sc + RT * EA);                    // [E]: this block's tokens per expert, then its base
    md_pdl_launch_dependents();
    md_pdl_wait();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int t0 = blockIdx.x * RT, n = min(RT, rows - t0);
    for (int e = tid; e < E; e += RW * 32) cnt[e] = 0;
    const __nv_bfloat16* lo = h + (size_t)(t0 + min(g, n - 1)) * W + t * 8;
    const __nv_bfloat16* hi = h + (size_t)(t0 + min(g + 8, n - 1)) * W + t * 8;
    for (int e0 = 0; e0 < EA; e0 += RE) {
        float acc[RE / 8][4];
#pragma unroll
        for (int i = 0; i < RE / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll 2
        for (int k = warp * 32; k < W; k += RW * 32) {
            const bool live = k + t * 8 < W;      // W % 8 == 0
            const uint4 z = make_uint4(0, 0, 0, 0), a = live ? ld_act(lo + k) : z, b = live ? ld_act(hi + k) : z;
#pragma unroll
            for (int i = 0; i < RE / 8; ++i) {
                const int e = e0 + i * 8 + g;
                if (e0 + i * 8 >= EA) break;
                const uint4 x = live && e < EA ? *reinterpret_cast<const uint4*>(router + (size_t)e * W + t * 8 + k) : z;
                mma_piece(acc[i], a, b, x);
            }
        }
#pragma unroll
        for (int i = 0; i < RE / 8; ++i) {
            part[warp][g][i * 8 + 2 * t] = acc[i][0];
            part[warp][g][i * 8 + 2 * t + 1] = acc[i][1];
            part[warp][g + 8][i * 8 + 2 * t] = acc[i][2];
            part[warp][g + 8][i * 8 + 2 * t + 1] = acc[i][3];
        }
        __syncthreads();
        for (int i = tid; i < RT * RE; i += RW * 32) {
            const int r = i / RE, e = i % RE;
            float v = 0.f;
#pragma unroll
            for (int w = 0; w < RW; ++w) v += part[w][r][e];
            if (e0 + e < EA) sc[r * EA + e0 + e] = v;
        }
        __syncthreads();
    }
    for (int r = warp; r < n; r += RW)
        warp_top(sc + r * EA, E, top, kind, lane, [&](int k, int e, float v) {
            const size_t at = (size_t)(t0 + r) * top + k;
            score[(size_t)(t0 + r) * (top + shared) + k] = v;
            sel[at] = e;
            rank[at] = atomicAdd(cnt + e, 1);
            if (k == 0 && shared) score[(size_t)(t0 + r) * (top + 1) + top] = md_logistic(sc[r * EA + E]);
        });
    __syncthreads();
    for (int e = tid; e < E; e += RW * 32)
        if (cnt[e]) cnt[e] = atomicAdd(count + e, cnt[e]);
    __syncthreads();
    for (int i = tid; i < n * top; i += RW * 32) {   // this block wrote sel and rank of its tokens
        const size_t at = (size_t)t0 * top + i;
        rank[at] += cnt[sel[at]];
    }
}

// ---- up to eight tokens
struct Route {
    float* score;        // [8][rows of the router]
    float* weight;       // [slots][8]
    float* shared;       // [8] the shared expert's weight
    int *expert, *n_slots;
    unsigned* ticket;    // zero between launches
};

__global__ void __launch_bounds__(512)
moe_route_kernel(const __nv_bfloat16* h, const __nv_bfloat16* __restrict__ router, int T, int W, int E, int shared, int top, int kind,
                 Route r) {
    const int EA = E + shared;               // rows of the router
    extern __shared__ float sc[];            // last block: [8][EA] logits, then [8][EA] chosen weights
    __shared__ float partial[16][16][8];
    __shared__ int last_s;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int row0 = blockIdx.x * 16;
    const __nv_bfloat16* w_lo = router + (size_t)min(row0 + g, EA - 1) * W + t * 8;
    const __nv_bfloat16* w_hi = router + (size_t)min(row0 + g + 8, EA - 1) * W + t * 8;
    const __nv_bfloat16* x = h + (size_t)min(g, T - 1) * W + t * 8;
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    const uint4 zero = make_uint4(0, 0, 0, 0);
    md_pdl_launch_dependents();
    bool waited = false;
    for (int k0 = warp * 32; k0 < W; k0 += 4 * 512) {
        uint4 lo[4], hi[4], xv[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int k = k0 + u * 512;
            const bool live = k + t * 8 < W;
            lo[u] = live ? ldg_stream(w_lo + k) : zero;
            hi[u] = live ? ldg_stream(w_hi + k) : zero;
        }
        if (!waited) md_pdl_wait();
        waited = true;
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int k = k0 + u * 512;
            xv[u] = g < T && k + t * 8 < W ? ld_act(x + k) : zero;
        }
#pragma unroll
        for (int u = 0; u < 4; ++u) mma_piece(acc, lo[u], hi[u], xv[u]);
    }
    if (!waited) md_pdl_wait();
    partial[warp][g][2 * t] = acc[0];
    partial[warp][g][2 * t + 1] = acc[1];
    partial[warp][g + 8][2 * t] = acc[2];
    partial[warp][g + 8][2 * t + 1] = acc[3];
    __syncthreads();
    if (tid < 128) {
        const int m = tid >> 4, e = tid & 15;
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < 16; ++w) v += partial[w][e][m];
        if (m < T && row0 + e < EA) (gridDim.x == 1 ? sc : r.score)[m * EA + row0 + e] = v;
    }
    float* chosen = sc + 8 * EA;
    for (int i = tid; i < T * EA; i += 512) chosen[i] = 0.f;
    if (gridDim.x > 1) {
        __threadfence();
        __syncthreads();
        if (tid == 0) last_s = atomicAdd(r.ticket, 1u) == gridDim.x - 1;
        __syncthreads();
        if (!last_s) return;
        __threadfence();
        if (tid == 0) *r.ticket = 0u;
        for (int i = tid; i < T * EA; i += 512) sc[i] = __ldcg(r.score + i);
    }
    __syncthreads();
    if (shared && tid < 8) r.shared[tid] = tid < T ? md_logistic(sc[tid * EA + E]) : 0.f;
    if (warp < T) warp_top(sc + warp * EA, E, top, kind, lane, [&](int, int e, float v) { chosen[warp * EA + e] = v; });
    __syncthreads();
    if (warp == 0) {
        int slots = 0;
        for (int e0 = 0; e0 < E; e0 += 32) {
            const int e = e0 + lane;
            bool used = false;
            for (int m = 0; m < T; ++m) used |= e < E && chosen[m * EA + e] != 0.f;
            const unsigned b = __ballot_sync(0xffffffffu, used);
            if (used) {
                const int s = slots + __popc(b & ((1u << lane) - 1u));
                r.expert[s] = e;
                for (int m = 0; m < 8; ++m) r.weight[s * 8 + m] = m < T ? chosen[m * EA + e] : 0.f;
            }
            slots += __popc(b);
        }
        if (lane == 0) *r.n_slots = slots;
    }
}

struct FewShared {       // the shared expert's products; pad 0: none
    const __nv_bfloat16 *gu, *down;
    int pad;
    float limit;
};

// act[token][slot * ff_pad + j] = weight * gated(gate_j, up_j); the shared expert's columns follow those of all `slots`
__global__ void __launch_bounds__(256)
moe_up_kernel(const __nv_bfloat16* h, const __nv_bfloat16* __restrict__ w_gu, __nv_bfloat16* out, int T, int W, int ff_pad, int act,
              float limit, float alpha, int slots, FewShared sh, Route r) {
    __shared__ float partial[8][16][8];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int slot = blockIdx.y, j = blockIdx.x * 8 + g;
    md_pdl_launch_dependents();
    md_pdl_wait();
    // (the three small loads together; entries past n_slots are dropped right after)
    const bool is_shared = slot == slots;
    const float* weight = is_shared ? r.shared : r.weight + slot * 8;
    const int n_slots = __ldcg(r.n_slots), expert = is_shared ? 0 : __ldcg(r.expert + slot);
    const float mine = __ldcg(weight + g);
    if (is_shared ? (int)blockIdx.x * 8 >= sh.pad : slot >= n_slots || (int)blockIdx.x * 8 >= ff_pad) return;
    if (is_shared) limit = sh.limit;
    const __nv_bfloat16* w = is_shared ? sh.gu : w_gu + (size_t)expert * 2 * ff_pad * W;
    const __nv_bfloat16* w_lo = w + (size_t)((j / MD_GLU_BLOCK) * (2 * MD_GLU_BLOCK) + j % MD_GLU_BLOCK) * W + t * 8;
    const __nv_bfloat16* w_hi = w_lo + (size_t)MD_GLU_BLOCK * W;
    const bool has_x = g < T && mine != 0.f;
    const __nv_bfloat16* x = h + (size_t)(has_x ? g : 0) * W + t * 8;
    const uint4 zero = make_uint4(0, 0, 0, 0);
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    for (int k0 = warp * 32; k0 < W; k0 += 8 * 256) {
        uint4 lo[8], hi[8], xv[8];
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            const int k = k0 + u * 256;
            const bool live = k + t * 8 < W;
            lo[u] = live ? ldg_stream(w_lo + k) : zero;
            hi[u] = live ? ldg_stream(w_hi + k) : zero;
            xv[u] = live && has_x ? ld_act(x + k) : zero;
        }
#pragma unroll
        for (int u = 0; u < 8; ++u) mma_piece(acc, lo[u], hi[u], xv[u]);
    }
    partial[warp][g][2 * t] = acc[0];
    partial[warp][g][2 * t + 1] = acc[1];
    partial[warp][g + 8][2 * t] = acc[2];
    partial[warp][g + 8][2 * t + 1] = acc[3];
    __syncthreads();
    if (tid < 64) {
        const int m = tid >> 3, e = tid & 7;
        if (m < T) {
            float a = 0.f, b = 0.f;
#pragma unroll
            for (int q = 0; q < 8; ++q) {
                a += partial[q][e][m];
                b += partial[q][e + 8][m];
            }
            out[(size_t)m * (slots * ff_pad + sh.pad) + slot * ff_pad + blockIdx.x * 8 + e] =
                __float2bfloat16_rn(__ldcg(weight + m) * md_gated(act, limit, alpha, a, b));
        }
    }
}

// y[token][n] = sum over the slots' columns
__global__ void __launch_bounds__(512, 2)
moe_down_kernel(const __nv_bfloat16* act, const __nv_bfloat16* __restrict__ w_down, float* y, int T, int W, int ff_pad, int slots,
                FewShared sh, Route r) {
    __shared__ float partial[16][16][8];
    __shared__ int list[MAX_EXPERTS];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int row0 = blockIdx.x * 16, per = ff_pad / 32, act_stride = slots * ff_pad + sh.pad;
    md_pdl_launch_dependents();
    md_pdl_wait();
    const int n_slots = __ldcg(r.n_slots), routed = n_slots * per, chunks = routed + sh.pad / 32;
    if (tid < slots) list[tid] = __ldcg(r.expert + tid);   // what is past n_slots is not used
    __syncthreads();
    const size_t r_lo = min(row0 + g, W - 1), r_hi = min(row0 + g + 8, W - 1);
    const __nv_bfloat16* x = act + (size_t)(g < T ? g : 0) * act_stride + t * 8;
    const uint4 zero = make_uint4(0, 0, 0, 0);
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    constexpr int U = 4;
    for (int c0 = warp; c0 < chunks; c0 += U * 16) {
        uint4 lo[U], hi[U], xv[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int c = c0 + u * 16;
            lo[u] = hi[u] = xv[u] = zero;
            if (c < chunks) {
                const bool own = c < routed;
                const int slot = own ? c / per : 0, pitch = own ? ff_pad : sh.pad;
                const __nv_bfloat16* w = own ? w_down + (size_t)list[slot] * W * ff_pad + (c - slot * per) * 32 : sh.down + (c - routed) * 32;
                lo[u] = ldg_stream(w + r_lo * pitch + t * 8);
                hi[u] = ldg_stream(w + r_hi * pitch + t * 8);
                if (g < T) xv[u] = ld_act(x + (own ? c * 32 : slots * ff_pad + (c - routed) * 32));
            }
        }
#pragma unroll
        for (int u = 0; u < U; ++u) mma_piece(acc, lo[u], hi[u], xv[u]);
    }
    partial[warp][g][2 * t] = acc[0];
    partial[warp][g][2 * t + 1] = acc[1];
    partial[warp][g + 8][2 * t] = acc[2];
    partial[warp][g + 8][2 * t + 1] = acc[3];
    __syncthreads();
    if (tid < 128) {
        const int m = tid >> 4, e = tid & 15;
        if (m < T && row0 + e < W) {
            float v = 0.f;
#pragma unroll
            for (int w = 0; w < 16; ++w) v += partial[w][e][m];
            y[(size_t)m * W + row0 + e] = v;
        }
    }
}

int launch_few(md_ctx* ctx, const md_moe& m, const void* h, size_t rows, const md_moe_buffers& b) {
    const int T = (int)rows, E = m.experts, EA = E + (m.shared_pad > 0), slots = T * m.top < E ? T * m.top : E;
    Route r;
    // the ticket first: layers of different sizes share the buffer, and it must stay what the last launch left, zero
    r.ticket = reinterpret_cast<unsigned*>(b.route);
    r.n_slots = reinterpret_cast<int*>(b.route) + 1;
    r.shared = b.route + 8;
    r.score = r.shared + 8;
    r.weight = r.score + 8 * (size_t)EA;
    r.expert = reinterpret_cast<int*>(r.weight + 8 * (size_t)EA);
    const FewShared sh = {reinterpret_cast<const __nv_bfloat16*>(m.shared_gu), reinterpret_cast<const __nv_bfloat16*>(m.shared_down),
                          m.shared_pad, m.shared_limit};
    const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(h);
    __nv_bfloat16* act = reinterpret_cast<__nv_bfloat16*>(b.act);
    MD_TRY(md_launch_ex(ctx, moe_route_kernel, dim3((unsigned)((EA + 15) / 16)), dim3(512), 16 * (size_t)EA * sizeof(float), "moe_route_kernel",
                        x, reinterpret_cast<const __nv_bfloat16*>(m.router), T, m.width, E, EA - E, m.top, m.router_kind, r));
    MD_TRY(md_launch_ex(ctx, moe_up_kernel, dim3((unsigned)((m.ff_pad > m.shared_pad ? m.ff_pad : m.shared_pad) / 8), (unsigned)(slots + EA - E)),
                        dim3(256), 0, "moe_up_kernel", x,
                        reinterpret_cast<const __nv_bfloat16*>(m.w_gu), act, T, m.width, m.ff_pad, m.act, m.limit, m.alpha,
                        slots, sh, r));
    return md_launch_ex(ctx, moe_down_kernel, dim3((unsigned)((m.width + 15) / 16)), dim3(512), 0, "moe_down_kernel", act,
                        reinterpret_cast<const __nv_bfloat16*>(m.w_down), b.y_f32, T, m.width, m.ff_pad, slots, sh, r);
}

template <class T>
int launch_sorted(md_ctx* ctx, int dtype, const md_moe& m, const void* h, size_t rows, const md_moe_buffers& b) {
    const int shared = m.shared_pad > 0 ? 1 : 0;
    const size_t cap = md_moe_sorted_rows(rows, m.experts, m.top);
    MD_CUDA(ctx, cudaMemsetAsync(b.count, 0, m.experts * sizeof(int), ctx->stream));
    if (dtype == MD_DTYPE_BF16 && (m.width % 8) == 0) {
        const size_t smem = (RW * RT * RE + RT * (size_t)(m.experts + shared) + m.experts) * sizeof(float);
        if (smem > 48 * 1024)
            MD_CUDA(ctx, cudaFuncSetAttribute(moe_router_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        MD_TRY(md_launch_ex(ctx, moe_router_mma_kernel, dim3((unsigned)((rows + RT - 1) / RT)), dim3(RW * 32), smem, "moe_router_mma_kernel",
                            reinterpret_cast<const __nv_bfloat16*>(h), reinterpret_cast<const __nv_bfloat16*>(m.router), (int)rows,
                            m.width, m.experts, shared, m.top, m.router_kind, b.score, b.sel, b.rank, b.count));
    } else {
        MD_TRY(md_launch_ex(ctx, moe_router_kernel<T>, dim3((unsigned)((rows + 3) / 4)), dim3(128), 0, "moe_router_kernel",
                            reinterpret_cast<const T*>(h), reinterpret_cast<const T*>(m.router), (int)rows, m.width, m.experts,
                            shared, m.top, m.router_kind, b.score, b.sel, b.rank, b.count));
    }
    MD_TRY(md_launch_ex(ctx, moe_permute_kernel<T>, dim3((unsigned)rows), dim3(256), 0, "moe_permute_kernel",
                        reinterpret_cast<const T*>(h), m.width, m.experts, shared ? (int)cap : -1, m.top, b.sel, b.rank, b.count, b.slot,
                        b.tile_expert, b.n_blocks, reinterpret_cast<T*>(b.xs)));
    md_lin up;
    up.glu = m.act, up.glu_limit = m.limit, up.glu_alpha = m.alpha;
    up.tile_expert = b.tile_expert;
    up.n_blocks = b.n_blocks;
    up.n_experts = m.experts;
    MD_TRY(md_linear(ctx, dtype, b.xs, m.w_gu, b.act, cap, 2 * (size_t)m.ff_pad, m.width, up));
    md_lin down = up;
    down.glu = 0;
    MD_TRY(md_linear(ctx, dtype, b.act, m.w_down, b.ys, cap, m.width, m.ff_pad, down));
    if (!shared) return MD_OK;
    md_lin own;
    own.glu = m.act, own.glu_limit = m.shared_limit, own.glu_alpha = m.alpha;
    MD_TRY(md_linear(ctx, dtype, h, m.shared_gu, b.shared_act, rows, 2 * (size_t)m.shared_pad, m.width, own));
    return md_linear(ctx, dtype, b.shared_act, m.shared_down, reinterpret_cast<T*>(b.ys) + cap * m.width, rows, m.width, m.shared_pad, md_lin());
}

}  // namespace

bool md_moe_sorted(int dtype, size_t width, size_t rows) {
    return dtype != MD_DTYPE_BF16 || (width % 8) != 0 || rows > 8;
}

size_t md_moe_sorted_rows(size_t rows, int experts, int top) {
    const size_t pairs = rows * top, used = pairs < (size_t)experts ? pairs : (size_t)experts;
    // every expert with a row wastes at most GROUP - 1 rows
    return (pairs + used * (MD_GROUP_ROWS - 1) + MD_GROUP_ROWS - 1) / MD_GROUP_ROWS * MD_GROUP_ROWS;
}

int md_launch_moe(md_ctx* ctx, int dtype, const md_moe& m, const void* h, size_t rows, const md_moe_buffers& b) {
    if (m.experts > MAX_EXPERTS || m.top > MAX_TOP || m.top > m.experts)
        return md_fail(ctx, MD_ERR_UNSUPPORTED, "mixture of experts: %d experts, %d per token", m.experts, m.top);
    if (!md_moe_sorted(dtype, m.width, rows)) return launch_few(ctx, m, h, rows, b);
    return dtype == MD_DTYPE_F32 ? launch_sorted<float>(ctx, dtype, m, h, rows, b)
                                 : launch_sorted<__nv_bfloat16>(ctx, dtype, m, h, rows, b);
}
