// Latent attention: all heads' keys and values are linear maps of one cached latent per token, beside a rotated key part that
// the heads share; sliding window and one sink logit per head (md_latent in stack.cuh).
//   rotation_table_kernel   (cos, sin) of every position
//   latent_norm_kernel      norms of the two latents, rotation of the shared key part, append to the cache
//   latent_plain_kernel     any element type and size, prompts and decoding: a block per (token, head) that takes the query
//                           into the latent space (q_h W_uk_h), so that scores and weighted sums run on the cached latents
//   latent_prefill_kernel   bfloat16 prompts: keys and values of the visible tokens come expanded from one product; 64 queries
//                           x 64 keys per step on tensor cores.  The query's rotation happens on its way to shared memory.
//                           Weights enter the second product as two bfloat16 terms (mma_bf16.cuh).
//   latent_heads_kernel     bfloat16, one token per sequence: per-head products (the query into the latent space, the weighted
//                           latent into the values), weights streamed as in gemv.cu
//   latent_decode_kernel    bfloat16, one token per sequence: 16 heads share every latent they read; the blocks of a cluster
//                           take parts of the window and merge through distributed shared memory
#include "mma_bf16.cuh"

#include <algorithm>

namespace {

constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
// 2^x by the hardware instruction (relative error about 2^-22), without exp2f's care for denormal results
__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

__global__ void rotation_table_kernel(float* table, int rows, int half, double base) {
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long long)rows * half) return;
    const int pos = (int)(i / half), k = (int)(i % half);
    double s, c;
    sincos((double)pos * pow(base, -(double)k / (double)half), &s, &c);
    table[2 * i] = (float)c;
    table[2 * i + 1] = (float)s;
}

template <class T, int V> __device__ __forceinline__ void load_v(const T* p, float (&f)[V]) {
    if constexpr (V == 4) md_load4<T>(p, f);
    else f[0] = md_elem<T>::get(*p);
}
template <class T, int V> __device__ __forceinline__ void store_v(T* p, const float (&f)[V]) {
    if constexpr (V == 4) md_store4<T>(p, f);
    else *p = md_elem<T>::put(f[0]);
}

constexpr int NORM_THREADS = 256;

// block = (row, sequence); V = 4: every size a multiple of 4
template <class T, int V>
__global__ void __launch_bounds__(NORM_THREADS)
latent_norm_kernel(const __grid_constant__ md_latent p) {
    extern __shared__ __align__(16) float xs[];   // the row
    __shared__ float red[2][NORM_THREADS / 32];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, t = blockIdx.x, seq = blockIdx.y;
    const int Q = p.q_rank, R = p.kv_rank, n = Q + R + p.rot;
    md_pdl_launch_dependents();
    md_pdl_wait();
    const int pos = (p.pos_dev[seq] ? *p.pos_dev[seq] : p.pos0) + t;
    const size_t row = (size_t)seq * p.rows + t;
    const T* in = reinterpret_cast<const T*>(p.in) + row * p.row_stride;
    float sq = 0.f, sc = 0.f;
    for (int c = tid * V; c < n; c += NORM_THREADS * V) {
        float f[V];
        load_v<T, V>(in + c, f);
#pragma unroll
        for (int i = 0; i < V; ++i) {
            xs[c + i] = f[i];
            if (c < Q) sq = fmaf(f[i], f[i], sq);
            else if (c < Q + R) sc = fmaf(f[i], f[i], sc);
        }
    }
    sq = warp_sum(sq);
    sc = warp_sum(sc);
    if (lane == 0) red[0][warp] = sq, red[1][warp] = sc;
    __syncthreads();
    sq = sc = 0.f;
#pragma unroll
    for (int i = 0; i < NORM_THREADS / 32; ++i) sq += red[0][i], sc += red[1][i];
    const float iq = 1.f / sqrtf(sq / (float)Q + p.eps), ic = 1.f / sqrtf(sc / (float)R + p.eps);
    T* cq = reinterpret_cast<T*>(p.cq) + row * Q;
    T* cc = reinterpret_cast<T*>(p.cc[seq]) + (size_t)pos * R;
    T* kr = reinterpret_cast<T*>(p.kr[seq]) + (size_t)pos * p.rot;
    for (int c = tid * V; c < Q + R; c += NORM_THREADS * V) {
        float w[V], f[V];
        load_v<float, V>(c < Q ? p.q_norm + c : p.kv_norm + (c - Q), w);
#pragma unroll
        for (int i = 0; i < V; ++i) f[i] = xs[c + i] * (c < Q ? iq : ic) * w[i];
        store_v<T, V>(c < Q ? cq + c : cc + (c - Q), f);
    }
    for (int i = tid; i < p.rot / 2; i += NORM_THREADS) {
        const float2 cs = *reinterpret_cast<const float2*>(p.rope + ((size_t)pos * (p.rot / 2) + i) * 2);
        const float u = xs[Q + R + 2 * i], v = xs[Q + R + 2 * i + 1];
        kr[2 * i] = md_elem<T>::put(u * cs.x - v * cs.y);
        kr[2 * i + 1] = md_elem<T>::put(v * cs.x + u * cs.y);
    }
}

constexpr int PLAIN_THREADS = 128;

// block x = token * heads + head, y = sequence
template <class T>
__global__ void __launch_bounds__(PLAIN_THREADS)
latent_plain_kernel(const __grid_constant__ md_latent p) {
    extern __shared__ __align__(16) float sm[];
    const int R = p.kv_rank, D = p.dim, rot = p.rot, H = p.heads;
    float* qa = sm;               // [R + rot] the query in the latent space, then its rotated part
    float* o = qa + R + rot;      // [R]
    float* q = o + R;             // [D]
    float* s = q + D;             // [PLAIN_THREADS]
    __shared__ float red[2][PLAIN_THREADS / 32];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, seq = blockIdx.y;
    const int t = blockIdx.x / H, h = blockIdx.x % H;
    md_pdl_launch_dependents();
    md_pdl_wait();
    const int pos = (p.pos_dev[seq] ? *p.pos_dev[seq] : p.pos0) + t;
    const T* qr = reinterpret_cast<const T*>(p.q) + ((size_t)seq * p.rows + t) * H * (D + rot) + (size_t)h * (D + rot);
    for (int i = tid; i < D; i += PLAIN_THREADS) q[i] = md_elem<T>::get(qr[i]);
    for (int i = tid; i < rot / 2; i += PLAIN_THREADS) {
        const float c = p.rope[((size_t)pos * (rot / 2) + i) * 2], sn = p.rope[((size_t)pos * (rot / 2) + i) * 2 + 1];
        const float u = md_elem<T>::get(qr[D + 2 * i]), v = md_elem<T>::get(qr[D + 2 * i + 1]);
        qa[R + 2 * i] = u * c - v * sn;
        qa[R + 2 * i + 1] = v * c + u * sn;
    }
    __syncthreads();
    const T* uk = reinterpret_cast<const T*>(p.w_ukv) + (size_t)h * D * R;
    for (int r = tid; r < R; r += PLAIN_THREADS) {
        float a = 0.f;
        for (int d = 0; d < D; ++d) a = fmaf(md_elem<T>::get(uk[(size_t)d * R + r]), q[d], a);
        qa[r] = a;
        o[r] = 0.f;
    }
    __syncthreads();
    const T* cc = reinterpret_cast<const T*>(p.cc[seq]);
    const T* kr = reinterpret_cast<const T*>(p.kr[seq]);
    float m = p.sink[h], l = 1.f;     // the sink: one more term of the denominator
    for (int k0 = p.window > 0 ? max(0, pos - p.window + 1) : 0; k0 <= pos; k0 += PLAIN_THREADS) {
        const int n = min(PLAIN_THREADS, pos - k0 + 1);
        for (int j = warp; j < n; j += PLAIN_THREADS / 32) {
            const T *cj = cc + (size_t)(k0 + j) * R, *kj = kr + (size_t)(k0 + j) * rot;
            float a = 0.f;
            for (int r = lane; r < R; r += 32) a = fmaf(qa[r], md_elem<T>::get(cj[r]), a);
            for (int r = lane; r < rot; r += 32) a = fmaf(qa[R + r], md_elem<T>::get(kj[r]), a);
            a = warp_sum(a);
            if (lane == 0) s[j] = a * p.scale;
        }
        __syncthreads();
        float mx = tid < n ? s[tid] : -INFINITY;
#pragma unroll
        for (int x = 16; x; x >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, x));
        if (lane == 0) red[0][warp] = mx;
        __syncthreads();
        float mn = m;
#pragma unroll
        for (int i = 0; i < PLAIN_THREADS / 32; ++i) mn = fmaxf(mn, red[0][i]);
        const float w = tid < n ? expf(s[tid] - mn) : 0.f, corr = expf(m - mn), ws = warp_sum(w);
        if (lane == 0) red[1][warp] = ws;
        s[tid] = w;
        __syncthreads();
        l *= corr;
#pragma unroll
        for (int i = 0; i < PLAIN_THREADS / 32; ++i) l += red[1][i];
        m = mn;
        for (int r = tid; r < R; r += PLAIN_THREADS) {
            float a = o[r] * corr;
            for (int j = 0; j < n; ++j) a = fmaf(s[j], md_elem<T>::get(cc[(size_t)(k0 + j) * R + r]), a);
            o[r] = a;
        }
        __syncthreads();
    }
    const T* uv = reinterpret_cast<const T*>(p.w_ukv) + ((size_t)H * D + (size_t)h * p.vdim) * R;
    T* out = reinterpret_cast<T*>(p.out) + (((size_t)seq * p.rows + t) * H + h) * p.vdim;
    for (int e = warp; e < p.vdim; e += PLAIN_THREADS / 32) {
        float a = 0.f;
        for (int r = lane; r < R; r += 32) a = fmaf(md_elem<T>::get(uv[(size_t)e * R + r]), o[r], a);
        a = warp_sum(a);
        if (lane == 0) out[e] = md_elem<T>::put(a / l);
    }
}

// ---- bfloat16 prompts
constexpr int BQ = 64, BK = 64, PRE_THREADS = 128;

// DK, DV: dim + rot and vdim rounded up (the pad is zero in shared memory)
template <int DK, int DV>
__global__ void __launch_bounds__(PRE_THREADS, DK + DV <= 160 ? 3 : DK + DV <= 320 ? 2 : 1)
latent_prefill_kernel(const __grid_constant__ md_latent p, int key0) {
    using namespace mb;
    constexpr int KP = DK + 8, VP = DV + 8;
    constexpr bool Q_REGS = DK <= 128;    // longer heads re-read their query fragments from shared memory
    extern __shared__ __align__(16) unsigned char smem[];
    __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(smem);    // [BQ][KP]
    __nv_bfloat16* Ks = Qs + BQ * KP;                               // two tiles [BK][KP]
    __nv_bfloat16* Vs = Ks + 2 * BK * KP;                           // two tiles [BK][VP]
    md_pdl_launch_dependents();
    md_pdl_wait();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int q0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * BQ, h = blockIdx.y;
    const int D = p.dim, rot = p.rot, E = p.vdim, per_q = p.heads * (D + rot), per_kv = p.heads * (D + E);
    const int rows = min(BQ, p.rows - q0);
    const __nv_bfloat16* qb = reinterpret_cast<const __nv_bfloat16*>(p.q) + (size_t)q0 * per_q + h * (D + rot);
    const __nv_bfloat16* kb = reinterpret_cast<const __nv_bfloat16*>(p.kv) + h * D;
    const __nv_bfloat16* vb = reinterpret_cast<const __nv_bfloat16*>(p.kv) + p.heads * D + h * E;
    const __nv_bfloat16* rb = reinterpret_cast<const __nv_bfloat16*>(p.kr[0]);
    const float scale = p.scale * LOG2E;
    const int P0 = p.pos0 + q0, last = P0 + rows - 1, window = p.window > 0 ? p.window : 0x3fffffff;
    const int start = max(0, P0 - window + 1), n_tiles = (last - start) / BK + 1;

    const int kc = DK / 8, vc = DV / 8, dc = D / 8, rc = rot / 8, ec = E / 8;
    auto load_tile = [&](int i) {
        const int k0 = start + i * BK;
        __nv_bfloat16 *K = Ks + (size_t)(i & 1) * BK * KP, *V = Vs + (size_t)(i & 1) * BK * VP;
        for (int j = tid; j < BK * kc; j += PRE_THREADS) {
            const int r = j / kc, c = j % kc, key = k0 + r;
            __nv_bfloat16* dst = K + r * KP + c * 8;
            if (key <= last && c < dc) cp_async16(smem_u32(dst), kb + (size_t)(key - key0) * per_kv + c * 8);
            else if (key <= last && c < dc + rc) cp_async16(smem_u32(dst), rb + (size_t)key * rot + (c - dc) * 8);
            else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
        for (int j = tid; j < BK * vc; j += PRE_THREADS) {
            const int r = j / vc, c = j % vc, key = k0 + r;
            __nv_bfloat16* dst = V + r * VP + c * 8;
            if (key <= last && c < ec) cp_async16(smem_u32(dst), vb + (size_t)(key - key0) * per_kv + c * 8);
            else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
        cp_async_commit();
    };
    for (int i = tid; i < BQ * kc; i += PRE_THREADS) {
        const int r = i / kc, c = i % kc;
        if (r < rows && c < dc) cp_async16(smem_u32(Qs + r * KP + c * 8), qb + (size_t)r * per_q + c * 8);
        else if (r >= rows || c >= dc + rc) *reinterpret_cast<uint4*>(Qs + r * KP + c * 8) = make_uint4(0, 0, 0, 0);
    }
    load_tile(0);
    for (int i = tid; i < rows * (rot / 2); i += PRE_THREADS) {
        const int r = i / (rot / 2), c = i % (rot / 2);
        const float2 cs = *reinterpret_cast<const float2*>(p.rope + ((size_t)(P0 + r) * (rot / 2) + c) * 2);
        const uint32_t uv = *reinterpret_cast<const uint32_t*>(qb + (size_t)r * per_q + D + 2 * c);
        const float u = __uint_as_float(uv << 16), v = __uint_as_float(uv & 0xffff0000u);
        *reinterpret_cast<uint32_t*>(Qs + r * KP + D + 2 * c) = md_pack_bf16(u * cs.x - v * cs.y, v * cs.x + u * cs.y);
    }
    uint32_t qf[Q_REGS ? DK / 16 : 1][4];
    float o[DV / 8][4];
#pragma unroll
    for (int i = 0; i < DV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    // the sink: one more term of the denominator, there from the start
    const float sink = p.sink[h] * LOG2E;
    float m_run[2] = {sink, sink}, l_run[2] = {1.f, 1.f};
    const int q_row = warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, q_col = (lane >> 4) * 8;

    for (int it = 0; it < n_tiles; ++it) {
        const int k0 = start + it * BK;
        cp_async_wait<0>();
        __syncthreads();                              // tile `it` is there, and nobody reads the other buffers any more
        if (it + 1 < n_tiles) load_tile(it + 1);      // in flight while this tile is worked on
        if (Q_REGS && it == 0) {
#pragma unroll
            for (int ks = 0; ks < DK / 16; ++ks) ldsm_x4(smem_u32(Qs + q_row * KP + ks * 16 + q_col), qf[Q_REGS ? ks : 0]);
        }
        const __nv_bfloat16 *K = Ks + (size_t)(it & 1) * BK * KP, *V = Vs + (size_t)(it & 1) * BK * VP;
        float s[BK / 8][4];
#pragma unroll
        for (int i = 0; i < BK / 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
#pragma unroll
        for (int ks = 0; ks < DK / 16; ++ks) {
            if (!Q_REGS) ldsm_x4(smem_u32(Qs + q_row * KP + ks * 16 + q_col), qf[0]);
            const uint32_t (&q)[4] = qf[Q_REGS ? ks : 0];
#pragma unroll
            for (int np = 0; np < BK / 16; ++np) {
                uint32_t b[4];
                ldsm_x4(smem_u32(K + (np * 16 + (lane & 7) + (lane >> 4) * 8) * KP + ks * 16 + ((lane >> 3) & 1) * 8), b);
                mma(s[2 * np], q[0], q[1], q[2], q[3], b[0], b[1]);
                mma(s[2 * np + 1], q[0], q[1], q[2], q[3], b[2], b[3]);
            }
        }
        const int i0 = P0 + warp * 16 + g;            // position of this thread's first query row
        const bool edge = k0 + BK - 1 > P0 || last - k0 >= window;   // some pair of the tile is not visible
        float mx[2] = {-INFINITY, -INFINITY}, corr[2], rs[2] = {0.f, 0.f};
#pragma unroll
        for (int nt = 0; nt < BK / 8; ++nt) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                float v = s[nt][e] * scale;
                if (edge) {
                    const int d = i0 + (e >> 1) * 8 - (k0 + nt * 8 + 2 * t + (e & 1));
                    if (d < 0 || d >= window) v = -INFINITY;
                }
                s[nt][e] = v;
                mx[e >> 1] = fmaxf(mx[e >> 1], v);
            }
        }
#pragma unroll
        for (int rr = 0; rr < 2; ++rr) {
            mx[rr] = fmaxf(mx[rr], __shfl_xor_sync(0xffffffffu, mx[rr], 1));
            mx[rr] = fmaxf(mx[rr], __shfl_xor_sync(0xffffffffu, mx[rr], 2));
            const float mn = fmaxf(m_run[rr], mx[rr]);   // finite: the sink is in it
            corr[rr] = ex2(m_run[rr] - mn);
            m_run[rr] = mn;
        }
#pragma unroll
        for (int nt = 0; nt < BK / 8; ++nt) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                s[nt][e] = ex2(s[nt][e] - m_run[e >> 1]);
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
            for (int i = 0; i < DV / 8; ++i) {
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
            for (int dp = 0; dp < DV / 16; ++dp) {
                uint32_t b[4];
                ldsm_x4_t(smem_u32(V + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * VP + dp * 16 + (lane >> 4) * 8), b);
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
        const float f = 1.f / l_run[rr];
        __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + ((size_t)(q0 + r) * p.heads + h) * E;
#pragma unroll
        for (int nt = 0; nt < DV / 8; ++nt)
            if (nt < ec) *reinterpret_cast<uint32_t*>(out + nt * 8 + 2 * t) = md_pack_bf16(o[nt][2 * rr] * f, o[nt][2 * rr + 1] * f);
    }
}

// ---- bfloat16 decoding: one token per sequence
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

// out[s][h][n] = sum_k w[h][n][k] x[s][h][k]; K % 8 == 0.  Strides in elements.
struct HeadsProduct {
    const __nv_bfloat16 *w, *x;
    __nv_bfloat16* out;
    int N, K, seqs;
    int x_seq, x_head, out_seq, out_head;
    // rot > 0: the first block of a head also turns x[s][h][K .. K + rot) into out[s][h][N .. N + rot)
    int rot;
    const float* rope;
    const int* pos[MD_STACK_MAX_SEQS];
};
constexpr int HEADS_WARPS = 4, HEADS_UNROLL = 4;

__global__ void __launch_bounds__(HEADS_WARPS * 32)
latent_heads_kernel(const __grid_constant__ HeadsProduct p) {
    __shared__ float partial[HEADS_WARPS][16][8];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int row0 = blockIdx.x * 16, h = blockIdx.y;
    const __nv_bfloat16* w = p.w + (size_t)h * p.N * p.K + t * 8;
    const __nv_bfloat16 *w_lo = w + (size_t)min(row0 + g, p.N - 1) * p.K, *w_hi = w + (size_t)min(row0 + g + 8, p.N - 1) * p.K;
    const bool has_x = g < p.seqs;
    const __nv_bfloat16* x = p.x + (size_t)(has_x ? g : 0) * p.x_seq + (size_t)h * p.x_head + t * 8;
    const uint4 zero = make_uint4(0, 0, 0, 0);
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    md_pdl_launch_dependents();
    bool waited = false;
    for (int k0 = warp * 32; k0 < p.K; k0 += HEADS_UNROLL * HEADS_WARPS * 32) {
        uint4 lo[HEADS_UNROLL], hi[HEADS_UNROLL], xv[HEADS_UNROLL];
#pragma unroll
        for (int u = 0; u < HEADS_UNROLL; ++u) {
            const int k = k0 + u * HEADS_WARPS * 32;
            const bool live = k + t * 8 < p.K;
            lo[u] = live ? ldg_stream(w_lo + k) : zero;
            hi[u] = live ? ldg_stream(w_hi + k) : zero;
        }
        if (!waited) md_pdl_wait();
        waited = true;
#pragma unroll
        for (int u = 0; u < HEADS_UNROLL; ++u) {
            const int k = k0 + u * HEADS_WARPS * 32;
            xv[u] = has_x && k + t * 8 < p.K ? ld_act(x + k) : zero;
        }
#pragma unroll
        for (int u = 0; u < HEADS_UNROLL; ++u) {
            mb::mma(acc, lo[u].x, hi[u].x, lo[u].y, hi[u].y, xv[u].x, xv[u].y);
            mb::mma(acc, lo[u].z, hi[u].z, lo[u].w, hi[u].w, xv[u].z, xv[u].w);
        }
    }
    if (!waited) md_pdl_wait();
    partial[warp][g][2 * t] = acc[0];
    partial[warp][g][2 * t + 1] = acc[1];
    partial[warp][g + 8][2 * t] = acc[2];
    partial[warp][g + 8][2 * t + 1] = acc[3];
    __syncthreads();
    const int m = tid >> 4, e = tid & 15;      // 128 threads: 8 sequences x 16 rows
    if (m < p.seqs && row0 + e < p.N) {
        float v = 0.f;
#pragma unroll
        for (int i = 0; i < HEADS_WARPS; ++i) v += partial[i][e][m];
        p.out[(size_t)m * p.out_seq + (size_t)h * p.out_head + row0 + e] = __float2bfloat16_rn(v);
    }
    if (blockIdx.x == 0)
        for (int i = tid; i < p.seqs * (p.rot / 2); i += HEADS_WARPS * 32) {
            const int s = i / (p.rot / 2), c = i % (p.rot / 2);
            const float2 cs = *reinterpret_cast<const float2*>(p.rope + ((size_t)*p.pos[s] * (p.rot / 2) + c) * 2);
            const uint32_t uv = __ldcg(reinterpret_cast<const uint32_t*>(p.x + (size_t)s * p.x_seq + (size_t)h * p.x_head + p.K + 2 * c));
            const float u = __uint_as_float(uv << 16), v = __uint_as_float(uv & 0xffff0000u);
            *reinterpret_cast<uint32_t*>(p.out + (size_t)s * p.out_seq + (size_t)h * p.out_head + p.N + 2 * c) =
                md_pack_bf16(u * cs.x - v * cs.y, v * cs.x + u * cs.y);
        }
}

constexpr int DEC_THREADS = 256, DEC_WARPS = 8, DEC_HEADS = 16, DEC_MAX_SPLITS = 8;

__device__ __forceinline__ void cluster_sync() {
    asm volatile("barrier.cluster.arrive.release.aligned;\nbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
// f32 at this block's shared-memory address `addr`, of the cluster's block `rank`
__device__ __forceinline__ float ld_peer(uint32_t addr, int rank) {
    uint32_t a;
    float v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(a) : "r"(addr), "r"(rank));
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(a) : "memory");
    return v;
}
__device__ __forceinline__ float2 ld_peer2(uint32_t addr, int rank) {
    uint32_t a;
    float2 v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(a) : "r"(addr), "r"(rank));
    asm volatile("ld.shared::cluster.v2.f32 {%0, %1}, [%2];" : "=f"(v.x), "=f"(v.y) : "r"(a) : "memory");
    return v;
}

__host__ __device__ constexpr int dec_pitch(int kv_rank, int rot) { return (kv_rank + rot + 31) / 32 * 32 + 8; }
template <int TK> constexpr size_t dec_smem(int kv_rank, int rot) {
    return ((size_t)(DEC_HEADS + 2 * TK) * dec_pitch(kv_rank, rot) + 2 * DEC_HEADS * (TK + 8)) * 2 +
           (2 * DEC_WARPS * DEC_HEADS + 2 * DEC_HEADS + DEC_MAX_SPLITS * DEC_HEADS) * sizeof(float);
}

// Grid (splits, groups of 16 heads, sequences), clusters of all splits.  A split takes every tile of TK visible latents that is
// congruent to it.  NT: output tiles of 8 latent values per warp, 64 * NT >= kv_rank.
template <int TK, int NT>
__global__ void __launch_bounds__(DEC_THREADS)
latent_decode_kernel(const __grid_constant__ md_latent p) {
    using namespace mb;
    constexpr int PP = TK + 8;
    extern __shared__ __align__(16) unsigned char smem[];
    const int R = p.kv_rank, rot = p.rot, pitch = dec_pitch(R, rot), steps = (pitch - 8) / 32;
    __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(smem);       // [16][pitch]
    __nv_bfloat16* Ks = Qs + DEC_HEADS * pitch;                        // two tiles [TK][pitch]; afterwards [16][R] f32
    __nv_bfloat16* Ps = Ks + 2 * TK * pitch;                           // [2][16][PP]: weights as two terms
    float* mxs = reinterpret_cast<float*>(Ps + 2 * DEC_HEADS * PP);    // [8][16] maxima
    float* sms = mxs + DEC_WARPS * DEC_HEADS;                          // [8][16] sums
    float* ml = sms + DEC_WARPS * DEC_HEADS;                           // [2][16] this block's maximum and sum
    float* fac = ml + 2 * DEC_HEADS;                                   // [8][16] factors of the cluster's blocks
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int split = blockIdx.x, splits = gridDim.x, h0 = blockIdx.y * DEC_HEADS, seq = blockIdx.z;
    const int heads = min(DEC_HEADS, p.heads - h0);
    const int pos = *p.pos_dev[seq];      // written by the kernel that ended the previous step
    const int first = p.window > 0 ? max(0, pos - p.window + 1) : 0;
    const int tiles = (pos - first) / TK + 1, mine = split < tiles ? (tiles - split - 1) / splits + 1 : 0;
    const __nv_bfloat16* cc = reinterpret_cast<const __nv_bfloat16*>(p.cc[seq]);
    const __nv_bfloat16* kr = reinterpret_cast<const __nv_bfloat16*>(p.kr[seq]);
    const int ch = (pitch - 8) / 8, cr = R / 8, crot = (R + rot) / 8;
    md_pdl_launch_dependents();
    // keys [lo, hi) of tile `i` of this split; the other rows of the tile and its pad become zero with `fill`
    auto load_tile = [&](int i, int lo, int hi, bool fill) {
        const int k0 = first + (split + i * splits) * TK;
        __nv_bfloat16* K = Ks + (size_t)(i & 1) * TK * pitch;
        for (int j = tid; j < TK * ch; j += DEC_THREADS) {
            const int r = j / ch, c = j % ch, key = k0 + r;
            __nv_bfloat16* dst = K + r * pitch + c * 8;
            if (key >= lo && key < hi && c < crot)
                cp_async16(smem_u32(dst), c < cr ? cc + (size_t)key * R + c * 8 : kr + (size_t)key * rot + (c - cr) * 8);
            else if (fill && (key > pos || c >= crot))
                *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
    };
    // the cached latents of earlier steps are requested before the wait for this step's
    if (mine > 0) load_tile(0, 0, pos, true);
    cp_async_commit();
    md_pdl_wait();
    if (mine == 1) load_tile(0, pos, pos + 1, false);
    const __nv_bfloat16* qa = reinterpret_cast<const __nv_bfloat16*>(p.qa) + ((size_t)seq * p.heads + h0) * (R + rot);
    for (int j = tid; j < DEC_HEADS * ch; j += DEC_THREADS) {
        const int r = j / ch, c = j % ch;
        *reinterpret_cast<uint4*>(Qs + r * pitch + c * 8) =
            r < heads && c < crot ? ld_act(qa + (size_t)r * (R + rot) + c * 8) : make_uint4(0, 0, 0, 0);
    }
    cp_async_commit();

    const float scale = p.scale * LOG2E;
    float o[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};   // heads g and g + 8; sums over this thread's keys only
    constexpr int S_WARPS = TK / 8;      // warps that take a tile of 8 keys each
    const int a_row = (lane & 7) + ((lane >> 3) & 1) * 8, a_col = (lane >> 4) * 8;
    for (int it = 0; it < mine; ++it) {
        cp_async_wait<0>();
        __syncthreads();                 // tile `it` is there, and nobody reads the other buffer or the weights any more
        if (it + 1 < mine) load_tile(it + 1, 0, pos + 1, true);
        cp_async_commit();
        const __nv_bfloat16* K = Ks + (size_t)(it & 1) * TK * pitch;
        const int k0 = first + (split + it * splits) * TK;
        float s[4] = {0.f, 0.f, 0.f, 0.f};
        if (warp < S_WARPS) {
            float s2[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
            for (int ks = 0; ks < steps; ++ks) {
                uint32_t a0[4], a1[4], b[4];
                ldsm_x4(smem_u32(K + (warp * 8 + (lane & 7)) * pitch + ks * 32 + (lane >> 3) * 8), b);
                ldsm_x4(smem_u32(Qs + a_row * pitch + ks * 32 + a_col), a0);
                ldsm_x4(smem_u32(Qs + a_row * pitch + ks * 32 + 16 + a_col), a1);
                mma(s, a0[0], a0[1], a0[2], a0[3], b[0], b[1]);
                mma(s2, a1[0], a1[1], a1[2], a1[3], b[2], b[3]);
            }
            float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
            for (int e = 0; e < 4; ++e) {      // head g + 8 (e >> 1), key 2 t + (e & 1)
                s[e] = k0 + warp * 8 + 2 * t + (e & 1) <= pos ? (s[e] + s2[e]) * scale : -INFINITY;
                mx[e >> 1] = fmaxf(mx[e >> 1], s[e]);
            }
#pragma unroll
            for (int rr = 0; rr < 2; ++rr) {
                mx[rr] = fmaxf(mx[rr], __shfl_xor_sync(0xffffffffu, mx[rr], 1));
                mx[rr] = fmaxf(mx[rr], __shfl_xor_sync(0xffffffffu, mx[rr], 2));
                if (t == 0) mxs[warp * DEC_HEADS + g + 8 * rr] = mx[rr];
            }
        }
        __syncthreads();
        float corr[2];
#pragma unroll
        for (int rr = 0; rr < 2; ++rr) {
            float mn = m_run[rr];        // every tile holds a visible key: finite from here on
#pragma unroll
            for (int i = 0; i < S_WARPS; ++i) mn = fmaxf(mn, mxs[i * DEC_HEADS + g + 8 * rr]);
            corr[rr] = m_run[rr] == -INFINITY ? 0.f : ex2(m_run[rr] - mn);
            m_run[rr] = mn;
            l_run[rr] *= corr[rr];
        }
        if (warp < S_WARPS) {
#pragma unroll
            for (int rr = 0; rr < 2; ++rr) {
                const float w0 = ex2(s[2 * rr] - m_run[rr]), w1 = ex2(s[2 * rr + 1] - m_run[rr]);
                l_run[rr] += w0 + w1;
                uint32_t hi, lo;
                split2(w0, w1, hi, lo);
                __nv_bfloat16* dst = Ps + (g + 8 * rr) * PP + warp * 8 + 2 * t;
                *reinterpret_cast<uint32_t*>(dst) = hi;
                *reinterpret_cast<uint32_t*>(dst + DEC_HEADS * PP) = lo;
            }
        }
#pragma unroll
        for (int i = 0; i < NT; ++i) {
            o[i][0] *= corr[0]; o[i][1] *= corr[0];
            o[i][2] *= corr[1]; o[i][3] *= corr[1];
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < TK / 16; ++kk) {
            uint32_t hi[4], lo[4];
            ldsm_x4(smem_u32(Ps + a_row * PP + kk * 16 + a_col), hi);
            ldsm_x4(smem_u32(Ps + (DEC_HEADS + a_row) * PP + kk * 16 + a_col), lo);
#pragma unroll
            for (int np = 0; np < NT / 2; ++np) {
                const int col = (warp * NT + 2 * np) * 8;
                if (col >= R) break;
                uint32_t b[4];
                ldsm_x4_t(smem_u32(K + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * pitch + col + (lane >> 4) * 8), b);
                mma(o[2 * np], hi[0], hi[1], hi[2], hi[3], b[0], b[1]);
                mma(o[2 * np + 1], hi[0], hi[1], hi[2], hi[3], b[2], b[3]);
                mma(o[2 * np], lo[0], lo[1], lo[2], lo[3], b[0], b[1]);
                mma(o[2 * np + 1], lo[0], lo[1], lo[2], lo[3], b[2], b[3]);
            }
        }
    }
    cp_async_wait<0>();
#pragma unroll
    for (int rr = 0; rr < 2; ++rr) {
        l_run[rr] += __shfl_xor_sync(0xffffffffu, l_run[rr], 1);
        l_run[rr] += __shfl_xor_sync(0xffffffffu, l_run[rr], 2);
        if (t == 0) sms[warp * DEC_HEADS + g + 8 * rr] = l_run[rr];
        if (t == 0 && warp == 0) ml[g + 8 * rr] = m_run[rr];
    }
    __syncthreads();                     // all reads of the tiles are over
    float* Of = reinterpret_cast<float*>(Ks);
    if (mine > 0) {
#pragma unroll
        for (int i = 0; i < NT; ++i) {
            const int col = (warp * NT + i) * 8 + 2 * t;
            if (col >= R) break;
            *reinterpret_cast<float2*>(Of + g * R + col) = make_float2(o[i][0], o[i][1]);
            *reinterpret_cast<float2*>(Of + (g + 8) * R + col) = make_float2(o[i][2], o[i][3]);
        }
    }
    if (tid < DEC_HEADS) {
        float l = 0.f;
#pragma unroll
        for (int i = 0; i < DEC_WARPS; ++i) l += sms[i * DEC_HEADS + tid];
        ml[DEC_HEADS + tid] = l;
    }
    cluster_sync();
    if (tid < DEC_HEADS) {
        const uint32_t at = smem_u32(ml + tid);
        const float sink = p.sink[h0 + min(tid, heads - 1)] * LOG2E;
        float m = sink, pm[DEC_MAX_SPLITS], l;
#pragma unroll
        for (int i = 0; i < DEC_MAX_SPLITS; ++i) {
            pm[i] = i < splits ? ld_peer(at, i) : -INFINITY;
            m = fmaxf(m, pm[i]);
        }
        l = ex2(sink - m);
#pragma unroll
        for (int i = 0; i < DEC_MAX_SPLITS; ++i) {
            pm[i] = pm[i] == -INFINITY ? 0.f : ex2(pm[i] - m);
            if (i < splits) l = fmaf(ld_peer(at + DEC_HEADS * sizeof(float), i), pm[i], l);
        }
#pragma unroll
        for (int i = 0; i < DEC_MAX_SPLITS; ++i) fac[i * DEC_HEADS + tid] = pm[i] / l;
    }
    __syncthreads();
    __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.ol) + ((size_t)seq * p.heads + h0) * R;
    const int used = min(splits, tiles);
    for (int i = (split * DEC_THREADS + tid) * 2; i < heads * R; i += splits * DEC_THREADS * 2) {
        const int hh = i / R;
        const uint32_t at = smem_u32(Of + i);
        float2 a = make_float2(0.f, 0.f);
#pragma unroll
        for (int j = 0; j < DEC_MAX_SPLITS; ++j) {
            if (j >= used) break;
            const float2 v = ld_peer2(at, j);
            const float f = fac[j * DEC_HEADS + hh];
            a.x = fmaf(v.x, f, a.x);
            a.y = fmaf(v.y, f, a.y);
        }
        *reinterpret_cast<uint32_t*>(out + i) = md_pack_bf16(a.x, a.y);
    }
    cluster_sync();                      // the peers' shared memory stays until all have read it
}

bool eights(std::initializer_list<int> v) {
    for (int x : v)
        if (x % 8) return false;
    return true;
}
bool vector_ok(const md_latent& a) {
    return eights({a.dim, a.rot, a.vdim, a.q_rank, a.kv_rank, a.row_stride}) && a.dim + a.rot <= 256 && a.vdim <= 256;
}
bool decode_ok(const md_latent& a) { return vector_ok(a) && a.kv_rank <= 1024 && a.rot <= 256 && a.w_ukt; }

template <class T>
int launch_norm(md_ctx* ctx, const md_latent& a) {
    const size_t smem = (size_t)(a.q_rank + a.kv_rank + a.rot) * sizeof(float);
    if (smem > 200 * 1024) return md_fail(ctx, MD_ERR_UNSUPPORTED, "latent attention: latents of %d and %d values", a.q_rank, a.kv_rank);
    const bool v4 = ((a.q_rank | a.kv_rank | a.rot | a.row_stride) % 4) == 0;
    auto kern = v4 ? latent_norm_kernel<T, 4> : latent_norm_kernel<T, 1>;
    if (smem > 47 * 1024) MD_CUDA(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    return md_launch_ex(ctx, kern, dim3((unsigned)a.rows, (unsigned)a.seqs), dim3(NORM_THREADS), smem, "latent_norm_kernel", a);
}

template <class T>
int launch_plain(md_ctx* ctx, const md_latent& a) {
    const size_t smem = (size_t)(2 * a.kv_rank + a.rot + a.dim + PLAIN_THREADS) * sizeof(float);
    if (smem > 200 * 1024) return md_fail(ctx, MD_ERR_UNSUPPORTED, "latent attention: latent of %d values", a.kv_rank);
    if (smem > 47 * 1024)
        MD_CUDA(ctx, cudaFuncSetAttribute(latent_plain_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    return md_launch_ex(ctx, latent_plain_kernel<T>, dim3((unsigned)(a.rows * a.heads), (unsigned)a.seqs), dim3(PLAIN_THREADS), smem,
                        "latent_plain_kernel", a);
}

template <int DK, int DV>
int launch_prefill_as(md_ctx* ctx, const md_latent& a, int key0) {
    constexpr size_t smem = ((size_t)(BQ + 2 * BK) * (DK + 8) + 2 * BK * (DV + 8)) * 2;
    auto kern = latent_prefill_kernel<DK, DV>;
    MD_CUDA(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    return md_launch_ex(ctx, kern, dim3((unsigned)((a.rows + BQ - 1) / BQ), (unsigned)a.heads), dim3(PRE_THREADS), smem,
                        "latent_prefill_kernel", a, key0);
}

int launch_prefill(md_ctx* ctx, const md_latent& a) {
    const int key0 = a.window > 0 ? std::max(0, a.pos0 - a.window + 1) : 0, keys = a.pos0 + a.rows - key0;
    const size_t R = a.kv_rank;
    MD_TRY(md_linear(ctx, MD_DTYPE_BF16, reinterpret_cast<const __nv_bfloat16*>(a.cc[0]) + key0 * R, a.w_ukv, a.kv, keys,
                     (size_t)a.heads * (a.dim + a.vdim), R, md_lin()));
    const int dk = a.dim + a.rot, dv = a.vdim;
    if (dk <= 64 && dv <= 64) return launch_prefill_as<64, 64>(ctx, a, key0);
    if (dk <= 96 && dv <= 64) return launch_prefill_as<96, 64>(ctx, a, key0);
    if (dk <= 128 && dv <= 64) return launch_prefill_as<128, 64>(ctx, a, key0);
    if (dk <= 128 && dv <= 128) return launch_prefill_as<128, 128>(ctx, a, key0);
    if (dk <= 192 && dv <= 128) return launch_prefill_as<192, 128>(ctx, a, key0);
    return launch_prefill_as<256, 256>(ctx, a, key0);
}

int launch_heads(md_ctx* ctx, const HeadsProduct& h, int heads) {
    return md_launch_ex(ctx, latent_heads_kernel, dim3((unsigned)((h.N + 15) / 16), (unsigned)heads), dim3(HEADS_WARPS * 32), 0,
                        "latent_heads_kernel", h);
}

template <int TK, int NT>
int launch_decode_as(md_ctx* ctx, const md_latent& a) {
    const size_t most = md_latent_keys(1, a.window > 0 ? a.window : 0, a.max_seq), tiles = (most + TK - 1) / TK;
    const unsigned splits = (unsigned)std::min<size_t>(DEC_MAX_SPLITS, tiles);
    const size_t smem = dec_smem<TK>(a.kv_rank, a.rot);
    auto kern = latent_decode_kernel<TK, NT>;
    MD_CUDA(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(splits, (unsigned)((a.heads + DEC_HEADS - 1) / DEC_HEADS), (unsigned)a.seqs);
    cfg.blockDim = dim3(DEC_THREADS);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = ctx->stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = splits;
    attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = ctx->pdl ? 2 : 1;
    const cudaError_t e = cudaLaunchKernelEx(&cfg, kern, a);
    if (e != cudaSuccess) return md_fail(ctx, MD_ERR_CUDA, "launch of latent_decode_kernel failed: %s", cudaGetErrorString(e));
    ctx->launches++;
    return MD_OK;
}

int launch_decode(md_ctx* ctx, const md_latent& a) {
    const int D = a.dim, R = a.kv_rank, rot = a.rot, H = a.heads;
    const __nv_bfloat16* ukv = reinterpret_cast<const __nv_bfloat16*>(a.w_ukv);
    HeadsProduct q = {};
    q.w = reinterpret_cast<const __nv_bfloat16*>(a.w_ukt), q.x = reinterpret_cast<const __nv_bfloat16*>(a.q);
    q.out = reinterpret_cast<__nv_bfloat16*>(a.qa);
    q.N = R, q.K = D, q.seqs = a.seqs;
    q.x_seq = H * (D + rot), q.x_head = D + rot, q.out_seq = H * (R + rot), q.out_head = R + rot;
    q.rot = rot, q.rope = a.rope;
    for (int i = 0; i < a.seqs; ++i) q.pos[i] = a.pos_dev[i];
    MD_TRY(launch_heads(ctx, q, H));
    if (R <= 128) MD_TRY((launch_decode_as<64, 2>(ctx, a)));
    else if (R <= 256) MD_TRY((launch_decode_as<64, 4>(ctx, a)));
    else if (R <= 512) MD_TRY((launch_decode_as<64, 8>(ctx, a)));
    else MD_TRY((launch_decode_as<32, 16>(ctx, a)));
    HeadsProduct v = {};
    v.w = ukv + (size_t)H * D * R, v.x = reinterpret_cast<const __nv_bfloat16*>(a.ol), v.out = reinterpret_cast<__nv_bfloat16*>(a.out);
    v.N = a.vdim, v.K = R, v.seqs = a.seqs;
    v.x_seq = H * R, v.x_head = R, v.out_seq = H * a.vdim, v.out_head = a.vdim;
    return launch_heads(ctx, v, H);
}

}  // namespace

bool md_latent_expands(int dtype, const md_latent& a) { return dtype == MD_DTYPE_BF16 && vector_ok(a) && a.rows > 1 && a.seqs == 1; }

int md_launch_rotation_table(md_ctx* ctx, float* table, size_t rows, size_t dims, float base) {
    const long long n = (long long)rows * (dims / 2);
    if (n == 0) return MD_OK;
    rotation_table_kernel<<<(unsigned)((n + 255) / 256), 256, 0, ctx->stream>>>(table, (int)rows, (int)(dims / 2), (double)base);
    MD_LAUNCH_CHECK(ctx, "rotation_table_kernel");
    return MD_OK;
}

int md_launch_latent_attention(md_ctx* ctx, int dtype, const md_latent& a, bool decode) {
    const bool f32 = dtype == MD_DTYPE_F32;
    MD_TRY(f32 ? launch_norm<float>(ctx, a) : launch_norm<__nv_bfloat16>(ctx, a));
    const size_t rows = (size_t)a.rows * a.seqs;
    MD_TRY(md_linear(ctx, dtype, a.cq, a.w_uq, a.q, rows, (size_t)a.heads * (a.dim + a.rot), a.q_rank, md_lin()));
    if (md_latent_expands(dtype, a) && !decode) return launch_prefill(ctx, a);
    if (!f32 && decode && a.rows == 1 && decode_ok(a)) return launch_decode(ctx, a);
    return f32 ? launch_plain<float>(ctx, a) : launch_plain<__nv_bfloat16>(ctx, a);
}
