// Latent attention: all heads' keys and values are linear maps of one cached latent per token, beside a rotated key part that
// the heads share; sliding window and one sink logit per head (md_latent in stack.cuh).
//   rotation_table_kernel   (cos, sin) of every position
//   latent_norm_kernel      norms of the two latents, rotation of the shared key part, append to the cache
//   latent_plain_kernel     any element type and size, prompts and decoding: a block per (token, head) that takes the query
//                           into the latent space (q_h W_uk_h), so that scores and weighted sums run on the cached latents
//   latent_prefill_kernel   bfloat16 prompts whose head sizes the tcgen05 kernel (attention_latent_tc.cu) cannot hold: keys and
//                           values of the visible tokens come expanded from one product; 64 queries x 64 keys per step on
//                           mma.sync.  The query's rotation happens on its way to shared memory.  Weights enter the second
//                           product as two bfloat16 terms (mma_bf16.cuh).
//   latent_query_kernel     bfloat16, one token per sequence: norms, the queries' product and the append to the cache
//   latent_absorb_kernel    bfloat16, one token per sequence: the query into the latent space, per head
//   latent_decode_kernel    bfloat16, one token per sequence: 16 heads share every latent they read; blocks take parts of the
//                           window
//   latent_value_kernel     bfloat16, one token per sequence: merges the parts (and the sink), the weighted latent into the values
#include "mma_bf16.cuh"
#include "tc_common.cuh"

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
    if constexpr (V == 8) {
        const uint4 u = __ldcg(reinterpret_cast<const uint4*>(p));
        const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) f[2 * i] = __uint_as_float(w[i] << 16), f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    } else if constexpr (V == 4) {
        md_load4<T>(p, f);
    } else {
        f[0] = md_elem<T>::get(*p);
    }
}
template <int V> __device__ __forceinline__ void load_weight(const float* p, float (&f)[V]) {
    if constexpr (V == 1) {
        f[0] = __ldg(p);
    } else {
#pragma unroll
        for (int i = 0; i < V; i += 4) {
            const float4 v = __ldg(reinterpret_cast<const float4*>(p + i));
            f[i] = v.x, f[i + 1] = v.y, f[i + 2] = v.z, f[i + 3] = v.w;
        }
    }
}
template <class T, int V> __device__ __forceinline__ void store_v(T* p, const float (&f)[V]) {
    if constexpr (V == 8) {
        *reinterpret_cast<uint4*>(p) = make_uint4(md_pack_bf16(f[0], f[1]), md_pack_bf16(f[2], f[3]), md_pack_bf16(f[4], f[5]), md_pack_bf16(f[6], f[7]));
    } else if constexpr (V == 4) {
        md_store4<T>(p, f);
    } else {
        *p = md_elem<T>::put(f[0]);
    }
}

constexpr int NORM_WARPS = 4;

// a warp per row, y = sequence; V divides every size
template <class T, int V>
__global__ void __launch_bounds__(NORM_WARPS * 32)
latent_norm_kernel(const __grid_constant__ md_latent p) {
    const int lane = threadIdx.x & 31, t = blockIdx.x * NORM_WARPS + (threadIdx.x >> 5), seq = blockIdx.y;
    const int Q = p.q_rank, R = p.kv_rank;
    md_pdl_launch_dependents();
    md_pdl_wait();
    if (t >= p.rows) return;
    const int pos = (p.pos_dev[seq] ? *p.pos_dev[seq] : p.pos0) + t;
    const size_t row = (size_t)seq * p.rows + t;
    const T* in = reinterpret_cast<const T*>(p.in) + row * p.row_stride;
    constexpr int KEEP = 48 / V;     // vectors of a latent that stay in registers; the second pass finds the others in L2
    float q[KEEP][V], k[KEEP][V];
    auto load = [&](const T* src, int n, float (&f)[KEEP][V]) {
#pragma unroll
        for (int j = 0; j < KEEP; ++j)
            if ((lane + 32 * j) * V < n) load_v<T, V>(src + (lane + 32 * j) * V, f[j]);
    };
    auto norm = [&](const T* src, int n, const float* w, T* dst, float (&f)[KEEP][V]) {
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < KEEP; ++j) {
#pragma unroll
            for (int i = 0; i < V; ++i)
                if ((lane + 32 * j) * V < n) ss = fmaf(f[j][i], f[j][i], ss);
        }
        for (int c = (lane + 32 * KEEP) * V; c < n; c += 32 * V) {
            float x[V];
            load_v<T, V>(src + c, x);
#pragma unroll
            for (int i = 0; i < V; ++i) ss = fmaf(x[i], x[i], ss);
        }
        const float inv = 1.f / sqrtf(warp_sum(ss) / (float)n + p.eps);
        auto put = [&](int c, float (&x)[V]) {
            float g[V];
            load_weight<V>(w + c, g);
#pragma unroll
            for (int i = 0; i < V; ++i) x[i] *= inv * g[i];
            store_v<T, V>(dst + c, x);
        };
#pragma unroll
        for (int j = 0; j < KEEP; ++j)
            if ((lane + 32 * j) * V < n) put((lane + 32 * j) * V, f[j]);
        for (int c = (lane + 32 * KEEP) * V; c < n; c += 32 * V) {
            float x[V];
            load_v<T, V>(src + c, x);
            put(c, x);
        }
    };
    load(in, Q, q);
    load(in + Q, R, k);
    norm(in, Q, p.q_norm, reinterpret_cast<T*>(p.cq) + row * Q, q);
    norm(in + Q, R, p.kv_norm, reinterpret_cast<T*>(p.cc[seq]) + (size_t)pos * R, k);
    T* kr = reinterpret_cast<T*>(p.kr[seq]) + (size_t)pos * p.rot;
    for (int i = lane; i < p.rot / 2; i += 32) {
        const float2 cs = *reinterpret_cast<const float2*>(p.rope + ((size_t)pos * (p.rot / 2) + i) * 2);
        const float u = md_elem<T>::get(in[Q + R + 2 * i]), v = md_elem<T>::get(in[Q + R + 2 * i + 1]);
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
    extern __shared__ __align__(128) unsigned char smem[];
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

// The query in the latent space: qa[s][h][r] = sum_d w_ukt[h][r][d] q[s][h][d]; the first block of a head also rotates the rotated
// part behind it.
constexpr int HEADS_WARPS = 4;

__global__ void __launch_bounds__(HEADS_WARPS * 32)
latent_absorb_kernel(const __grid_constant__ md_latent p) {
    __shared__ float partial[HEADS_WARPS][16][8];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int R = p.kv_rank, D = p.dim, rot = p.rot, row0 = blockIdx.x * 16, h = blockIdx.y;
    const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(p.w_ukt) + (size_t)h * R * D + t * 8;
    const __nv_bfloat16 *w_lo = w + (size_t)min(row0 + g, R - 1) * D, *w_hi = w + (size_t)min(row0 + g + 8, R - 1) * D;
    const bool has_x = g < p.seqs;
    const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(p.q) + (size_t)h * (D + rot);   // of sequence 0
    const int q_seq = p.heads * (D + rot);
    const __nv_bfloat16* x = q + (size_t)(has_x ? g : 0) * q_seq + t * 8;
    __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.qa) + (size_t)h * (R + rot);
    const int out_seq = p.heads * (R + rot);
    const uint4 zero = make_uint4(0, 0, 0, 0);
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    md_pdl_launch_dependents();
    constexpr int U = 2;               // head sizes up to 256
    uint4 lo[U], hi[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
        const int k = warp * 32 + u * HEADS_WARPS * 32;
        const bool live = k + t * 8 < D;
        lo[u] = live ? ldg_stream(w_lo + k) : zero;
        hi[u] = live ? ldg_stream(w_hi + k) : zero;
    }
    md_pdl_wait();
#pragma unroll
    for (int u = 0; u < U; ++u) {
        const int k = warp * 32 + u * HEADS_WARPS * 32;
        const uint4 xv = has_x && k + t * 8 < D ? ld_act(x + k) : zero;
        mb::mma(acc, lo[u].x, hi[u].x, lo[u].y, hi[u].y, xv.x, xv.y);
        mb::mma(acc, lo[u].z, hi[u].z, lo[u].w, hi[u].w, xv.z, xv.w);
    }
    partial[warp][g][2 * t] = acc[0];
    partial[warp][g][2 * t + 1] = acc[1];
    partial[warp][g + 8][2 * t] = acc[2];
    partial[warp][g + 8][2 * t + 1] = acc[3];
    __syncthreads();
    const int m = tid >> 4, e = tid & 15;      // 128 threads: 8 sequences x 16 rows
    if (m < p.seqs && row0 + e < R) {
        float v = 0.f;
#pragma unroll
        for (int i = 0; i < HEADS_WARPS; ++i) v += partial[i][e][m];
        out[(size_t)m * out_seq + row0 + e] = __float2bfloat16_rn(v);
    }
    if (blockIdx.x == 0)
        for (int i = tid; i < p.seqs * (rot / 2); i += HEADS_WARPS * 32) {
            const int s = i / (rot / 2), c = i % (rot / 2);
            const float2 cs = *reinterpret_cast<const float2*>(p.rope + ((size_t)*p.pos_dev[s] * (rot / 2) + c) * 2);
            const uint32_t uv = __ldcg(reinterpret_cast<const uint32_t*>(q + (size_t)s * q_seq + D + 2 * c));
            const float u = __uint_as_float(uv << 16), v = __uint_as_float(uv & 0xffff0000u);
            *reinterpret_cast<uint32_t*>(out + (size_t)s * out_seq + R + 2 * c) = md_pack_bf16(u * cs.x - v * cs.y, v * cs.x + u * cs.y);
        }
}

// The start of a decode step: blocks x < rows / 16 compute q = w_uq cq with cq = rms(in[0 .. q_rank); q_norm) normed on the way
// (the norm's factor is a number per token, applied to the sums), the last block of a sequence norms and rotates the new token's
// latent and appends it to the cache.
constexpr int UQ_WARPS = 8, UQ_UNROLL = 4;

__global__ void __launch_bounds__(UQ_WARPS * 32)
latent_query_kernel(const __grid_constant__ md_latent p, int row_blocks) {
    __shared__ float partial[UQ_WARPS][16][8], red[UQ_WARPS][8];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int Q = p.q_rank, R = p.kv_rank, rot = p.rot;
    md_pdl_launch_dependents();
    if ((int)blockIdx.x >= row_blocks) {
        const int seq = blockIdx.x - row_blocks, pos = *p.pos_dev[seq];   // written by the kernel that ended the previous step
        const __nv_bfloat16* in = reinterpret_cast<const __nv_bfloat16*>(p.in) + (size_t)seq * p.row_stride + Q;
        md_pdl_wait();
        float ss = 0.f;
        for (int c = tid * 4; c < R; c += UQ_WARPS * 32 * 4) {
            float f[4];
            md_load4<__nv_bfloat16>(in + c, f);
#pragma unroll
            for (int i = 0; i < 4; ++i) ss = fmaf(f[i], f[i], ss);
        }
        ss = warp_sum(ss);
        if (lane == 0) red[warp][0] = ss;
        __syncthreads();
        ss = 0.f;
#pragma unroll
        for (int i = 0; i < UQ_WARPS; ++i) ss += red[i][0];
        const float inv = 1.f / sqrtf(ss / (float)R + p.eps);
        __nv_bfloat16* cc = reinterpret_cast<__nv_bfloat16*>(p.cc[seq]) + (size_t)pos * R;
        for (int c = tid * 4; c < R; c += UQ_WARPS * 32 * 4) {
            float f[4], w[4];
            md_load4<__nv_bfloat16>(in + c, f);
            md_load4<float>(p.kv_norm + c, w);
#pragma unroll
            for (int i = 0; i < 4; ++i) f[i] *= inv * w[i];
            md_store4<__nv_bfloat16>(cc + c, f);
        }
        for (int i = tid; i < rot / 2; i += UQ_WARPS * 32) {
            const float2 cs = *reinterpret_cast<const float2*>(p.rope + ((size_t)pos * (rot / 2) + i) * 2);
            const uint32_t uv = __ldcg(reinterpret_cast<const uint32_t*>(in + R + 2 * i));
            const float u = __uint_as_float(uv << 16), v = __uint_as_float(uv & 0xffff0000u);
            reinterpret_cast<uint32_t*>(reinterpret_cast<__nv_bfloat16*>(p.kr[seq]) + (size_t)pos * rot)[i] =
                md_pack_bf16(u * cs.x - v * cs.y, v * cs.x + u * cs.y);
        }
        return;
    }
    const int N = p.heads * (p.dim + rot), row0 = blockIdx.x * 16;
    const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(p.w_uq) + t * 8;
    const __nv_bfloat16 *w_lo = w + (size_t)min(row0 + g, N - 1) * Q, *w_hi = w + (size_t)min(row0 + g + 8, N - 1) * Q;
    const bool has_x = g < p.seqs;
    const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(p.in) + (size_t)(has_x ? g : 0) * p.row_stride + t * 8;
    const float* nw = p.q_norm + t * 8;
    const uint4 zero = make_uint4(0, 0, 0, 0);
    float acc[4] = {0.f, 0.f, 0.f, 0.f}, ss = 0.f;
    bool waited = false;
    for (int k0 = warp * 32; k0 < Q; k0 += UQ_UNROLL * UQ_WARPS * 32) {
        uint4 lo[UQ_UNROLL], hi[UQ_UNROLL], xv[UQ_UNROLL];
        float4 n0[UQ_UNROLL], n1[UQ_UNROLL];
#pragma unroll
        for (int u = 0; u < UQ_UNROLL; ++u) {
            const int k = k0 + u * UQ_WARPS * 32;
            const bool live = k + t * 8 < Q;
            lo[u] = live ? ldg_stream(w_lo + k) : zero;
            hi[u] = live ? ldg_stream(w_hi + k) : zero;
            n0[u] = n1[u] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (live) {
                n0[u] = __ldg(reinterpret_cast<const float4*>(nw + k));
                n1[u] = __ldg(reinterpret_cast<const float4*>(nw + k) + 1);
            }
        }
        if (!waited) md_pdl_wait();
        waited = true;
#pragma unroll
        for (int u = 0; u < UQ_UNROLL; ++u) {
            const int k = k0 + u * UQ_WARPS * 32;
            xv[u] = has_x && k + t * 8 < Q ? ld_act(x + k) : zero;
        }
#pragma unroll
        for (int u = 0; u < UQ_UNROLL; ++u) {
            const uint32_t v[4] = {xv[u].x, xv[u].y, xv[u].z, xv[u].w};
            const float f[8] = {n0[u].x, n0[u].y, n0[u].z, n0[u].w, n1[u].x, n1[u].y, n1[u].z, n1[u].w};
            uint32_t b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float a0 = __uint_as_float(v[i] << 16), a1 = __uint_as_float(v[i] & 0xffff0000u);
                ss = fmaf(a0, a0, fmaf(a1, a1, ss));
                b[i] = md_pack_bf16(a0 * f[2 * i], a1 * f[2 * i + 1]);
            }
            mb::mma(acc, lo[u].x, hi[u].x, lo[u].y, hi[u].y, b[0], b[1]);
            mb::mma(acc, lo[u].z, hi[u].z, lo[u].w, hi[u].w, b[2], b[3]);
        }
    }
    if (!waited) md_pdl_wait();
    ss += __shfl_xor_sync(0xffffffffu, ss, 1);
    ss += __shfl_xor_sync(0xffffffffu, ss, 2);
    if (t == 0) red[warp][g] = ss;
    partial[warp][g][2 * t] = acc[0];
    partial[warp][g][2 * t + 1] = acc[1];
    partial[warp][g + 8][2 * t] = acc[2];
    partial[warp][g + 8][2 * t + 1] = acc[3];
    __syncthreads();
    const int m = tid >> 4, e = tid & 15;
    if (tid < 128 && m < p.seqs && row0 + e < N) {
        float v = 0.f, s2 = 0.f;
#pragma unroll
        for (int i = 0; i < UQ_WARPS; ++i) v += partial[i][e][m], s2 += red[i][m];
        reinterpret_cast<__nv_bfloat16*>(p.q)[(size_t)m * N + row0 + e] = __float2bfloat16_rn(v / sqrtf(s2 / (float)Q + p.eps));
    }
}

constexpr int DEC_THREADS = 256, DEC_WARPS = 8, DEC_HEADS = 16, DEC_MAX_SPLITS = 32;

__device__ __forceinline__ void bulk_load(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst), "l"(src),
                 "r"(bytes), "r"(bar)
                 : "memory");
}

// What the blocks of a window leave for latent_value_kernel: unnormalised sums and their (maximum, sum of weights).
struct LatentParts {
    float* o;        // [seqs][heads][splits][kv_rank]
    float2* ml;      // [seqs][heads][splits]
    int splits;      // blocks a window is dealt to; those past its last tile leave nothing
    int tile;        // latents per tile
    int buffers;     // 2 if a block may have more than one tile
};
__device__ __forceinline__ int visible_tiles(int pos, int window, int tile) {
    return (window > 0 ? min(pos, window - 1) : pos) / tile + 1;
}

__host__ __device__ constexpr int dec_pitch(int kv_rank, int rot) { return (kv_rank + rot + 31) / 32 * 32 + 8; }
template <int TK> constexpr size_t dec_smem(int kv_rank, int rot, int buffers) {
    return ((size_t)(DEC_HEADS + buffers * TK) * dec_pitch(kv_rank, rot) + 2 * DEC_HEADS * (TK + 8)) * 2 +
           (size_t)(DEC_WARPS * 32 / TK) * DEC_HEADS * (TK + 8) * sizeof(float);
}

// Grid (splits, groups of 16 heads, sequences).  Split i takes the tiles i, i + splits, .. of TK visible latents.  NT: output
// tiles of 8 latent values per warp, 64 * NT >= kv_rank.  Latents arrive by bulk copies into padded rows; those of earlier
// steps are requested before the dependency wait.
template <int TK, int NT>
__global__ void __launch_bounds__(DEC_THREADS)
latent_decode_kernel(const __grid_constant__ md_latent p, const LatentParts parts, md_devflags* flags) {
    using namespace mb;
    // scores: warps are GROUPS groups of 32 keys x SLICES slices of the latent
    constexpr int PP = TK + 8, GROUPS = TK / 32, SLICES = DEC_WARPS / GROUPS, KPL = TK / 16;
    extern __shared__ __align__(128) unsigned char smem[];
    __shared__ __align__(8) unsigned long long bars[3];               // two tiles, the queries
    __shared__ float corr_s[DEC_HEADS];
    __shared__ int abort_s;
    const int R = p.kv_rank, rot = p.rot, pitch = dec_pitch(R, rot), steps = (pitch - 8) / 16;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int split = blockIdx.x, splits = parts.splits, h0 = blockIdx.y * DEC_HEADS, seq = blockIdx.z;
    const int heads = min(DEC_HEADS, p.heads - h0);
    __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(smem);       // [16][pitch]
    __nv_bfloat16* Ks = Qs + DEC_HEADS * pitch;                        // [buffers][TK][pitch]
    __nv_bfloat16* Ps = Ks + (size_t)parts.buffers * TK * pitch;       // [2][16][PP]: weights as two terms
    float* Sx = reinterpret_cast<float*>(Ps + 2 * DEC_HEADS * PP);     // [SLICES][16][PP]: partial scores
    const int pos = *p.pos_dev[seq];      // written by the kernel that ended the previous step
    const int first = p.window > 0 ? max(0, pos - p.window + 1) : 0, tiles = visible_tiles(pos, p.window, TK);
    md_pdl_launch_dependents();
    if (split >= tiles) return;
    const int mine = (tiles - split - 1) / splits + 1;
    const uint32_t bar = smem_u32(bars), row_bytes = (uint32_t)(R + rot) * 2;
    const __nv_bfloat16* cc = reinterpret_cast<const __nv_bfloat16*>(p.cc[seq]);
    const __nv_bfloat16* kr = reinterpret_cast<const __nv_bfloat16*>(p.kr[seq]);
    auto tile_key = [&](int i) { return first + (split + i * splits) * TK; };
    auto load_row = [&](int i, int r) {
        const size_t key = tile_key(i) + r;
        const uint32_t dst = smem_u32(Ks + ((size_t)(i & 1) * TK + r) * pitch), b = bar + 8 * (i & 1);
        bulk_load(dst, cc + key * R, R * 2, b);
        if (rot) bulk_load(dst + R * 2, kr + key * rot, rot * 2, b);
    };
    // by warp 0: the rows of tile i below key `end` (the barrier counts all of the tile's)
    auto load_tile = [&](int i, int end) {
        const int n = min(TK, pos + 1 - tile_key(i));
        if (lane == 0) tc::mbar_expect_tx(bar + 8 * (i & 1), n * row_bytes);
        __syncwarp();
        for (int r = lane; r < min(n, end - tile_key(i)); r += 32) load_row(i, r);
    };
    if (warp == 0) {
        if (lane == 0) {
            abort_s = 0;
            for (int i = 0; i < 3; ++i) tc::mbar_init(bar + 8 * i, 1);
            asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        }
        __syncwarp();
        for (int i = 0; i < min(mine, 2); ++i) load_tile(i, pos);
        if (lane == 0) tc::mbar_expect_tx(bar + 16, heads * row_bytes);
        md_pdl_wait();
        // this step's latent, if one of the first tiles holds it, and the queries
        for (int i = 0; i < min(mine, 2); ++i)
            if (lane == 0 && pos - tile_key(i) < TK) load_row(i, pos - tile_key(i));
        if (lane < heads)
            bulk_load(smem_u32(Qs + lane * pitch),
                      reinterpret_cast<const __nv_bfloat16*>(p.qa) + ((size_t)seq * p.heads + h0 + lane) * (R + rot), row_bytes, bar + 16);
    } else {
        // what no copy fills: the pad of every row, heads and keys that are not there
        const uint4 zero = make_uint4(0, 0, 0, 0);
        const int pad0 = (R + rot) / 8, ch = (pitch - 8) / 8;
        for (int r = warp - 1; r < DEC_HEADS + min(mine, 2) * TK; r += DEC_WARPS - 1) {
            const int i = (r - DEC_HEADS) / TK;     // (rows of the queries: r < 16)
            const bool there = r < DEC_HEADS ? r < heads : tile_key(i) + (r - DEC_HEADS) % TK <= pos;
            for (int c = (there ? pad0 : 0) + lane; c < ch; c += 32) *reinterpret_cast<uint4*>(Qs + r * pitch + c * 8) = zero;
        }
    }
    __syncthreads();

    const float scale = p.scale * LOG2E;
    float o[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    float m_run = -INFINITY, l_run = 0.f;      // of head 2 * warp + (lane >> 4); the sum over this lane's keys only
    const int a_row = (lane & 7) + ((lane >> 3) & 1) * 8, a_col = (lane >> 4) * 8;
    const int b_row = (lane & 7) + (lane >> 4) * 8, b_col = ((lane >> 3) & 1) * 8;
    const int grp = warp % GROUPS, slice = warp / GROUPS, per = (steps + SLICES - 1) / SLICES;
    const int s_lo = slice * per, s_hi = min(steps, s_lo + per);
    const int sh = 2 * warp + (lane >> 4), sk = (lane & 15) * KPL;    // softmax: this lane's head and first key
    bool ok = tc::mbar_wait(bar + 16, 0, &abort_s, flags, 61);
    for (int it = 0; it < mine; ++it) {
        ok = tc::mbar_wait(bar + 8 * (it & 1), (it >> 1) & 1, &abort_s, flags, 62) && ok;
        const __nv_bfloat16* K = Ks + (size_t)(it & 1) * TK * pitch;
        {
            float s[4][4];
#pragma unroll
            for (int i = 0; i < 4; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
            const uint32_t qa = smem_u32(Qs + a_row * pitch + a_col), kb = smem_u32(K + (grp * 32 + b_row) * pitch + b_col);
#pragma unroll 3
            for (int ks = s_lo; ks < s_hi; ++ks) {
                uint32_t a[4], b0[4], b1[4];
                ldsm_x4(qa + ks * 32, a);
                ldsm_x4(kb + ks * 32, b0);
                ldsm_x4(kb + 32 * pitch + ks * 32, b1);
                mma(s[0], a[0], a[1], a[2], a[3], b0[0], b0[1]);
                mma(s[1], a[0], a[1], a[2], a[3], b0[2], b0[3]);
                mma(s[2], a[0], a[1], a[2], a[3], b1[0], b1[1]);
                mma(s[3], a[0], a[1], a[2], a[3], b1[2], b1[3]);
            }
            float* dst = Sx + (slice * DEC_HEADS + g) * PP + grp * 32 + 2 * t;
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                *reinterpret_cast<float2*>(dst + i * 8) = make_float2(s[i][0], s[i][1]);
                *reinterpret_cast<float2*>(dst + 8 * PP + i * 8) = make_float2(s[i][2], s[i][3]);
            }
        }
        __syncthreads();        // the scores are there, and nobody reads the previous tile any more
        if (it + 1 >= 2 && it + 1 < mine && warp == 0) {
            tc::fence_async_smem();
            load_tile(it + 1, pos + 1);
        }
        {
            float v[KPL];
#pragma unroll
            for (int i = 0; i < KPL; ++i) v[i] = 0.f;
#pragma unroll
            for (int c = 0; c < SLICES; ++c) {
                const float* src = Sx + (c * DEC_HEADS + sh) * PP + sk;
#pragma unroll
                for (int i = 0; i < KPL; i += 2) {
                    const float2 x = *reinterpret_cast<const float2*>(src + i);
                    v[i] += x.x;
                    v[i + 1] += x.y;
                }
            }
            float mx = -INFINITY;
#pragma unroll
            for (int i = 0; i < KPL; ++i) {
                v[i] = tile_key(it) + sk + i <= pos ? v[i] * scale : -INFINITY;
                mx = fmaxf(mx, v[i]);
            }
#pragma unroll
            for (int x = 8; x; x >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, x));
            const float mn = fmaxf(m_run, mx);       // every tile holds a visible key: finite
            const float corr = m_run == -INFINITY ? 0.f : ex2(m_run - mn);
            m_run = mn;
            l_run *= corr;
#pragma unroll
            for (int i = 0; i < KPL; i += 2) {
                const float w0 = ex2(v[i] - mn), w1 = ex2(v[i + 1] - mn);
                l_run += w0 + w1;
                uint32_t hi, lo;
                split2(w0, w1, hi, lo);
                *reinterpret_cast<uint32_t*>(Ps + sh * PP + sk + i) = hi;
                *reinterpret_cast<uint32_t*>(Ps + (DEC_HEADS + sh) * PP + sk + i) = lo;
            }
            if ((lane & 15) == 0) corr_s[sh] = corr;
        }
        __syncthreads();
        if (it > 0) {
            const float c0 = corr_s[g], c1 = corr_s[g + 8];
#pragma unroll
            for (int i = 0; i < NT; ++i) {
                o[i][0] *= c0; o[i][1] *= c0;
                o[i][2] *= c1; o[i][3] *= c1;
            }
        }
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
                ldsm_x4_t(smem_u32(K + (kk * 16 + a_row) * pitch + col + a_col), b);
                mma(o[2 * np], hi[0], hi[1], hi[2], hi[3], b[0], b[1]);
                mma(o[2 * np + 1], hi[0], hi[1], hi[2], hi[3], b[2], b[3]);
                mma(o[2 * np], lo[0], lo[1], lo[2], lo[3], b[0], b[1]);
                mma(o[2 * np + 1], lo[0], lo[1], lo[2], lo[3], b[2], b[3]);
            }
        }
    }
    if (!ok) return;                          // a copy did not arrive within the wait's limit: reported through `flags`
#pragma unroll
    for (int x = 8; x; x >>= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, x);
    const size_t slot = ((size_t)seq * p.heads + h0) * splits + split;   // + head * splits
    if ((lane & 15) == 0 && sh < heads) parts.ml[slot + (size_t)sh * splits] = make_float2(m_run, l_run);
    float* out = parts.o + (slot + (size_t)g * splits) * R;
#pragma unroll
    for (int i = 0; i < NT; ++i) {
        const int col = (warp * NT + i) * 8 + 2 * t;
        if (col >= R) break;
        if (g < heads) *reinterpret_cast<float2*>(out + col) = make_float2(o[i][0], o[i][1]);
        if (g + 8 < heads) *reinterpret_cast<float2*>(out + 8 * (size_t)splits * R + col) = make_float2(o[i][2], o[i][3]);
    }
}

// out[s][h][e] = sum_r w[h][e][r] o[s][h][r] with o merged from the window's parts, the sink in its denominator.  Block: 32 rows
// of a head, four sequences; 4 warps split the latent.
constexpr int VAL_THREADS = 256, VAL_UNROLL = 4, VAL_MAX_RANK = 1024, VAL_SEQS = 4;

__global__ void __launch_bounds__(VAL_THREADS)
latent_value_kernel(const __grid_constant__ md_latent p, const LatentParts parts) {
    __shared__ __align__(16) __nv_bfloat16 xs[VAL_SEQS][VAL_MAX_RANK + 8];
    __shared__ float fac[VAL_SEQS][DEC_MAX_SPLITS];
    __shared__ int used[VAL_SEQS];
    __shared__ float partial[4][32][9];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int R = p.kv_rank, E = p.vdim, h = blockIdx.y, row0 = blockIdx.x * 32 + (warp & 1) * 16, slice = warp >> 1;
    const int seq0 = blockIdx.z * VAL_SEQS, seqs = min(VAL_SEQS, p.seqs - seq0);
    const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(p.w_ukv) + ((size_t)p.heads * p.dim + (size_t)h * E) * R + t * 8;
    const __nv_bfloat16 *w_lo = w + (size_t)min(row0 + g, E - 1) * R, *w_hi = w + (size_t)min(row0 + g + 8, E - 1) * R;
    const uint4 zero = make_uint4(0, 0, 0, 0);
    md_pdl_launch_dependents();
    uint4 lo[VAL_UNROLL], hi[VAL_UNROLL];
    auto weights = [&](int k0) {
#pragma unroll
        for (int u = 0; u < VAL_UNROLL; ++u) {
            const int k = k0 + u * 128;
            const bool live = k + t * 8 < R;
            lo[u] = live ? ldg_stream(w_lo + k) : zero;
            hi[u] = live ? ldg_stream(w_hi + k) : zero;
        }
    };
    weights(slice * 32);
    if (warp < seqs && lane == 0) used[warp] = min(parts.splits, visible_tiles(*p.pos_dev[seq0 + warp], p.window, parts.tile));
    __syncwarp();
    md_pdl_wait();
    if (warp < seqs) {           // a warp per sequence, a lane per part
        const bool live = lane < used[warp];
        const float2 v = live ? __ldcg(parts.ml + ((size_t)(seq0 + warp) * p.heads + h) * parts.splits + lane) : make_float2(-INFINITY, 0.f);
        const float sink = p.sink[h] * LOG2E;
        float m = fmaxf(v.x, sink);
#pragma unroll
        for (int x = 16; x; x >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, x));
        const float f = live ? ex2(v.x - m) : 0.f, l = warp_sum(v.y * f) + ex2(sink - m);
        fac[warp][lane] = f / l;
    }
    __syncthreads();
    const int quads = R / 4;
    for (int i = tid; i < seqs * quads; i += VAL_THREADS) {
        const int s = i / quads, c = (i - s * quads) * 4, n = used[s];
        const float* src = parts.o + ((size_t)(seq0 + s) * p.heads + h) * parts.splits * R + c;
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
        for (int j = 0; j < n; ++j) {
            const float4 v = __ldcg(reinterpret_cast<const float4*>(src + (size_t)j * R));
            const float f = fac[s][j];
            a.x = fmaf(v.x, f, a.x); a.y = fmaf(v.y, f, a.y);
            a.z = fmaf(v.z, f, a.z); a.w = fmaf(v.w, f, a.w);
        }
        *reinterpret_cast<uint2*>(&xs[s][c]) = make_uint2(md_pack_bf16(a.x, a.y), md_pack_bf16(a.z, a.w));
    }
    __syncthreads();
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    const bool has_x = g < seqs;
    for (int k0 = slice * 32; k0 < R; k0 += VAL_UNROLL * 128) {
        if (k0 != slice * 32) weights(k0);
#pragma unroll
        for (int u = 0; u < VAL_UNROLL; ++u) {
            const int k = k0 + u * 128 + t * 8;
            const uint4 x = has_x && k < R ? *reinterpret_cast<const uint4*>(&xs[has_x ? g : 0][k]) : zero;
            mb::mma(acc, lo[u].x, hi[u].x, lo[u].y, hi[u].y, x.x, x.y);
            mb::mma(acc, lo[u].z, hi[u].z, lo[u].w, hi[u].w, x.z, x.w);
        }
    }
    float (*dst)[9] = partial[slice] + (warp & 1) * 16;
    dst[g][2 * t] = acc[0];
    dst[g][2 * t + 1] = acc[1];
    dst[g + 8][2 * t] = acc[2];
    dst[g + 8][2 * t + 1] = acc[3];
    __syncthreads();
    const int s = tid >> 5, e = blockIdx.x * 32 + lane;
    if (s < seqs && e < E)
        reinterpret_cast<__nv_bfloat16*>(p.out)[((size_t)(seq0 + s) * p.heads + h) * E + e] =
            __float2bfloat16_rn(partial[0][lane][s] + partial[1][lane][s] + partial[2][lane][s] + partial[3][lane][s]);
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
    constexpr int V = 16 / sizeof(T);
    auto kern = ((a.q_rank | a.kv_rank | a.row_stride) % V) == 0 ? latent_norm_kernel<T, V> : latent_norm_kernel<T, 1>;
    return md_launch_ex(ctx, kern, dim3((unsigned)((a.rows + NORM_WARPS - 1) / NORM_WARPS), (unsigned)a.seqs), dim3(NORM_WARPS * 32), 0,
                        "latent_norm_kernel", a);
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
    if (ctx->attn_tc != 0 && md_latent_tc_supported(a)) return md_launch_latent_tc(ctx, a, key0);
    if (a.dim + a.rot <= 128 && a.vdim <= 128) return launch_prefill_as<128, 128>(ctx, a, key0);
    return launch_prefill_as<256, 256>(ctx, a, key0);
}

template <int TK, int NT>
int launch_decode_as(md_ctx* ctx, const md_latent& a) {
    const size_t most = md_latent_keys(1, a.window > 0 ? a.window : 0, a.max_seq), tiles = (most + TK - 1) / TK;
    const size_t groups = (a.heads + DEC_HEADS - 1) / DEC_HEADS, rows = (size_t)a.seqs * a.heads;
    // a block per SM where the windows are long enough
    const size_t splits = std::max<size_t>(1, std::min<size_t>({DEC_MAX_SPLITS, tiles, ctx->sm_count / (a.seqs * groups)}));
    LatentParts parts;
    parts.splits = (int)splits, parts.tile = TK, parts.buffers = tiles > splits ? 2 : 1;
    void* scratch = nullptr;
    MD_TRY(md_scratch(ctx, rows * splits * (a.kv_rank * sizeof(float) + sizeof(float2)), &scratch));
    parts.o = reinterpret_cast<float*>(scratch);
    parts.ml = reinterpret_cast<float2*>(parts.o + rows * splits * a.kv_rank);
    const size_t smem = dec_smem<TK>(a.kv_rank, a.rot, parts.buffers);
    auto kern = latent_decode_kernel<TK, NT>;
    MD_CUDA(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    MD_TRY(md_launch_ex(ctx, kern, dim3((unsigned)splits, (unsigned)groups, (unsigned)a.seqs), dim3(DEC_THREADS), smem, "latent_decode_kernel",
                        a, parts, ctx->flags));
    return md_launch_ex(ctx, latent_value_kernel, dim3((unsigned)((a.vdim + 31) / 32), (unsigned)a.heads, (unsigned)((a.seqs + VAL_SEQS - 1) / VAL_SEQS)), dim3(VAL_THREADS), 0,
                        "latent_value_kernel", a, parts);
}

int launch_decode(md_ctx* ctx, const md_latent& a) {
    const int D = a.dim, R = a.kv_rank, rot = a.rot, H = a.heads;
    const int row_blocks = (H * (D + rot) + 15) / 16;
    MD_TRY(md_launch_ex(ctx, latent_query_kernel, dim3((unsigned)(row_blocks + a.seqs)), dim3(UQ_WARPS * 32), 0, "latent_query_kernel", a, row_blocks));
    MD_TRY(md_launch_ex(ctx, latent_absorb_kernel, dim3((unsigned)((R + 15) / 16), (unsigned)H), dim3(HEADS_WARPS * 32), 0, "latent_absorb_kernel", a));
    if (R <= 128) return launch_decode_as<64, 2>(ctx, a);
    if (R <= 256) return launch_decode_as<64, 4>(ctx, a);
    if (R <= 512) return launch_decode_as<64, 8>(ctx, a);
    return launch_decode_as<32, 16>(ctx, a);
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
    if (!f32 && decode && a.rows == 1 && decode_ok(a)) return launch_decode(ctx, a);
    MD_TRY(f32 ? launch_norm<float>(ctx, a) : launch_norm<__nv_bfloat16>(ctx, a));
    const size_t rows = (size_t)a.rows * a.seqs;
    MD_TRY(md_linear(ctx, dtype, a.cq, a.w_uq, a.q, rows, (size_t)a.heads * (a.dim + a.rot), a.q_rank, md_lin()));
    if (md_latent_expands(dtype, a) && !decode) return launch_prefill(ctx, a);
    return f32 ? launch_plain<float>(ctx, a) : launch_plain<__nv_bfloat16>(ctx, a);
}
