// What sits between the matrix products of a layer-stack decoder: residual update, RMS norms and the causal
// convolution in one kernel (md_glue in stack.cuh states the arithmetic), the append of new keys to a cache, and the
// greedy sample of f32 logits.  Everything is f32; only the row handed to the next product is rounded to T.
//   stack_glue_step_kernel   one row per sequence (a decode step, or the final norm of a few rows): a thread keeps its
//                            columns' inputs, weights and convolution state in registers, and all weights and the state are
//                            requested before the dependency wait
//   stack_glue_rows_kernel   rows of a prompt: a row per warp group, its inputs read once into registers
//   stack_glue_any_kernel    widths that are not a multiple of 4 or too wide for the others
//   stack_parallel_kernel    the same place in a layer whose two sublayers read the same row (md_parallel_glue): both layer
//                            scales and sums, one norm, two weighted outputs
#include "stack.cuh"

namespace {

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

__device__ __forceinline__ void prefetch_l2(const void* p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p)); }

template <int V> struct Vec { float f[V]; };
template <class T, int V> __device__ __forceinline__ Vec<V> ldv(const T* p) {
    Vec<V> r;
    if constexpr (V == 4) md_load4<T>(p, r.f);
    else r.f[0] = md_elem<T>::get(*p);
    return r;
}
// from shared memory (md_load4 reads global memory only)
template <int V> __device__ __forceinline__ Vec<V> lds(const float* p) {
    Vec<V> r;
    if constexpr (V == 4) {
        const float4 v = *reinterpret_cast<const float4*>(p);
        r.f[0] = v.x; r.f[1] = v.y; r.f[2] = v.z; r.f[3] = v.w;
    } else {
        r.f[0] = *p;
    }
    return r;
}
template <class T, int V> __device__ __forceinline__ void stv(T* p, const Vec<V>& v) {
    if constexpr (V == 4) md_store4<T>(p, v.f);
    else *p = md_elem<T>::put(v.f[0]);
}

// WIDE: all warps of the block work on one row at a time (a decode step has one row per sequence); otherwise one warp
// per row and as many rows as warps at once.  A block owns `R` rows of a sequence and recomputes the taps - 1 rows ahead
// of them; the first block of a sequence takes those from the state instead, and the last one, which then holds the
// sequence's last taps - 1 values of n (with older ones from the state if the sequence is that short), stores them.
template <class T, int V, bool WIDE>
__global__ void __launch_bounds__(WIDE ? 512 : 256)
stack_glue_any_kernel(const __grid_constant__ md_glue p, int R) {
    extern __shared__ __align__(16) float xs[];   // [R + halo][width]
    __shared__ float red[16];
    const int W = p.width, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int seq = blockIdx.y, t0 = blockIdx.x * R, own = min(R, p.rows - t0), halo = p.conv ? p.taps - 1 : 0;
    const bool first = blockIdx.x == 0;
    const int step = (WIDE ? blockDim.x : 32) * V, c0 = (WIDE ? tid : lane) * V;
    md_pdl_launch_dependents();
    md_pdl_wait();

    auto total = [&](float v) {
        v = warp_sum(v);
        if (WIDE) {
            if (lane == 0) red[warp] = v;
            __syncthreads();
            v = 0.f;
#pragma unroll
            for (int i = 0; i < 16; ++i) v += red[i];
            __syncthreads();
        }
        return v;
    };
    // n[t] of the sequence into xs[l]
    auto row = [&](int l, int t, bool store) {
        float* xr = xs + (size_t)l * W;
        const size_t g = (size_t)seq * p.rows + t, src = p.gather ? (size_t)p.gather[g] : g;
        float inv = 0.f;
        if (p.w_post) {
            float row_scale = 1.f, ss = 0.f;
            if (p.ssq) {
                float s = 0.f;
                for (int i = lane; i < p.ssq_parts; i += 32) s += p.ssq[src * p.ssq_parts + i];
                s = warp_sum(s);
                row_scale = 1.f / sqrtf(s / (float)p.ssq_n + p.eps);
            }
            for (int c = c0; c < W; c += step) {
                Vec<V> v;
                if (p.slot) {
#pragma unroll
                    for (int i = 0; i < V; ++i) v.f[i] = 0.f;
                    for (int k = 0; k < p.top; ++k) {
                        const float s = p.score[src * p.top + k];
                        const Vec<V> e = ldv<T, V>(reinterpret_cast<const T*>(p.y) + (size_t)p.slot[src * p.top + k] * W + c);
#pragma unroll
                        for (int i = 0; i < V; ++i) v.f[i] = fmaf(s, e.f[i], v.f[i]);
                    }
                } else if (p.y_f32) {
                    v = ldv<float, V>(p.y_f32 + src * W + c);
                } else {
                    v = ldv<T, V>(reinterpret_cast<const T*>(p.y) + src * W + c);
                }
#pragma unroll
                for (int i = 0; i < V; ++i) {
                    v.f[i] *= row_scale;
                    ss = fmaf(v.f[i], v.f[i], ss);
                }
                stv<float, V>(xr + c, v);
            }
            inv = p.mult / sqrtf(total(ss) / (float)W + p.eps);
        }
        float ss = 0.f;
        for (int c = c0; c < W; c += step) {
            Vec<V> v;
            if (p.tokens) {
                const unsigned long long tok = p.tokens[src];
                v = ldv<T, V>(reinterpret_cast<const T*>(p.embed) + (size_t)(tok < (unsigned long long)p.vocab ? tok : 0) * W + c);
            } else {
                v = ldv<float, V>(p.x + src * W + c);
            }
            if (p.w_post) {
                const Vec<V> y = lds<V>(xr + c), w = ldv<float, V>(p.w_post + c);
#pragma unroll
                for (int i = 0; i < V; ++i) v.f[i] = fmaf(y.f[i] * inv, w.f[i], v.f[i]);
            }
#pragma unroll
            for (int i = 0; i < V; ++i) ss = fmaf(v.f[i], v.f[i], ss);
            if (store && p.x_out) stv<float, V>(p.x_out + g * W + c, v);
            stv<float, V>(xr + c, v);
        }
        const float inv2 = 1.f / sqrtf(total(ss) / (float)W + p.eps);
        for (int c = c0; c < W; c += step) {
            Vec<V> v = lds<V>(xr + c);
            const Vec<V> w = ldv<float, V>(p.w_pre + c);
#pragma unroll
            for (int i = 0; i < V; ++i) v.f[i] *= inv2 * w.f[i];
            stv<float, V>(xr + c, v);
        }
    };

    const int slot = halo ? *p.state_slot[seq] : 0;
    float* state = halo ? p.state[seq] : nullptr;
    if (first && halo)
        for (int i = tid; i < halo * W; i += blockDim.x) xs[i] = state[slot * halo * W + i];
    const int lo = first ? halo : 0;
    if (WIDE) {
        for (int l = lo; l < halo + own; ++l) row(l, t0 - halo + l, l >= halo);
    } else {
        for (int l = lo + warp; l < halo + own; l += 8) row(l, t0 - halo + l, l >= halo);
    }
    __syncthreads();
    T* out = reinterpret_cast<T*>(p.out) + ((size_t)seq * p.rows + t0) * W;
    const int per = W / V;
    for (int i = tid; i < own * per; i += blockDim.x) {
        const int r = i / per, c = (i - r * per) * V;
        Vec<V> v = lds<V>(xs + (size_t)(r + halo) * W + c);
        if (p.conv) {
            Vec<V> s;
#pragma unroll
            for (int e = 0; e < V; ++e) s.f[e] = 0.f;
            for (int j = 0; j < p.taps; ++j) {
                const Vec<V> n = lds<V>(xs + (size_t)(r + j) * W + c), w = ldv<float, V>(p.conv + (size_t)j * W + c);
#pragma unroll
                for (int e = 0; e < V; ++e) s.f[e] = fmaf(w.f[e], n.f[e], s.f[e]);
            }
#pragma unroll
            for (int e = 0; e < V; ++e) v.f[e] += s.f[e];
        }
        stv<T, V>(out + (size_t)r * W + c, v);
    }
    if (blockIdx.x + 1 < gridDim.x || !halo) return;
    float* dst = state + (size_t)(p.rows == 1 ? slot : slot ^ 1) * halo * W;
    for (int i = tid; i < halo * W; i += blockDim.x) dst[i] = xs[(size_t)own * W + i];
}

constexpr int STEP_THREADS = 512;

// sum over the threads of a block of `WARPS` warps; red holds 2 * WARPS floats, `turn` alternates between its halves
template <int WARPS>
__device__ __forceinline__ float block_sum(float v, float* red, int turn) {
    v = warp_sum(v);
    float* r = red + turn * WARPS;
    if ((threadIdx.x & 31) == 0) r[threadIdx.x >> 5] = v;
    __syncthreads();
    v = 0.f;
#pragma unroll
    for (int i = 0; i < WARPS; ++i) v += r[i];
    return v;
}

// block x = row; width % 4 == 0, width <= 2048 * NV, taps <= TAPS
template <class T, int NV, int TAPS>
__global__ void __launch_bounds__(STEP_THREADS)
stack_glue_step_kernel(const __grid_constant__ md_glue p) {
    __shared__ float red[2 * STEP_THREADS / 32];
    const int W = p.width, tid = threadIdx.x, lane = tid & 31, row = blockIdx.x;
    md_pdl_launch_dependents();
    Vec<4> w_pre[NV], w_post[NV], conv[NV][TAPS], st[NV][TAPS - 1];
    const int halo = p.conv ? p.taps - 1 : 0;
    float* state = halo ? p.state[row] + (size_t)*p.state_slot[row] * halo * W : nullptr;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        const int c = (tid + n * STEP_THREADS) * 4;
        if (c >= W) continue;
        w_pre[n] = ldv<float, 4>(p.w_pre + c);
        if (p.w_post) w_post[n] = ldv<float, 4>(p.w_post + c);
#pragma unroll
        for (int j = 0; j < TAPS; ++j)
            if (p.conv && j < p.taps) conv[n][j] = ldv<float, 4>(p.conv + (size_t)j * W + c);
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j)
            if (j < halo) st[n][j] = ldv<float, 4>(state + (size_t)j * W + c);
    }
    md_pdl_wait();
    const size_t src = p.gather ? (size_t)p.gather[row] : row;
    Vec<4> x[NV], y[NV];
    const T* xe = p.tokens ? reinterpret_cast<const T*>(p.embed) +
                                 (size_t)(p.tokens[src] < (unsigned long long)p.vocab ? p.tokens[src] : 0ull) * W : nullptr;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        const int c = (tid + n * STEP_THREADS) * 4;
#pragma unroll
        for (int i = 0; i < 4; ++i) x[n].f[i] = y[n].f[i] = 0.f;
        if (c >= W) continue;
        x[n] = xe ? ldv<T, 4>(xe + c) : ldv<float, 4>(p.x + src * W + c);
        if (p.w_post && !p.slot) y[n] = p.y_f32 ? ldv<float, 4>(p.y_f32 + src * W + c) : ldv<T, 4>(reinterpret_cast<const T*>(p.y) + src * W + c);
    }
    if (p.w_post) {
        float scale = 1.f;
        if (p.ssq) {
            float s = 0.f;
            for (int i = lane; i < p.ssq_parts; i += 32) s += __ldcg(p.ssq + src * p.ssq_parts + i);
            scale = 1.f / sqrtf(warp_sum(s) / (float)p.ssq_n + p.eps);
        }
        if (p.slot)
            for (int k = 0; k < p.top; ++k) {
                const float s = p.score[src * p.top + k];
                const T* e = reinterpret_cast<const T*>(p.y) + (size_t)p.slot[src * p.top + k] * W;
#pragma unroll
                for (int n = 0; n < NV; ++n) {
                    const int c = (tid + n * STEP_THREADS) * 4;
                    if (c >= W) continue;
                    const Vec<4> v = ldv<T, 4>(e + c);
#pragma unroll
                    for (int i = 0; i < 4; ++i) y[n].f[i] = fmaf(s, v.f[i], y[n].f[i]);
                }
            }
        float ss = 0.f;
#pragma unroll
        for (int n = 0; n < NV; ++n) {
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                y[n].f[i] *= scale;
                ss = fmaf(y[n].f[i], y[n].f[i], ss);
            }
        }
        const float inv = p.mult / sqrtf(block_sum<STEP_THREADS / 32>(ss, red, 0) / (float)W + p.eps);
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            if ((tid + n * STEP_THREADS) * 4 >= W) continue;
#pragma unroll
            for (int i = 0; i < 4; ++i) x[n].f[i] = fmaf(y[n].f[i] * inv, w_post[n].f[i], x[n].f[i]);
        }
    }
    float ss = 0.f;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        const int c = (tid + n * STEP_THREADS) * 4;
#pragma unroll
        for (int i = 0; i < 4; ++i) ss = fmaf(x[n].f[i], x[n].f[i], ss);
        if (c < W && p.x_out) stv<float, 4>(p.x_out + (size_t)row * W + c, x[n]);
    }
    const float inv2 = 1.f / sqrtf(block_sum<STEP_THREADS / 32>(ss, red, 1) / (float)W + p.eps);
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        const int c = (tid + n * STEP_THREADS) * 4;
        if (c >= W) continue;
        Vec<4> v, o;
#pragma unroll
        for (int i = 0; i < 4; ++i) o.f[i] = v.f[i] = x[n].f[i] * (inv2 * w_pre[n].f[i]);
        if (p.conv) {
            Vec<4> s;
#pragma unroll
            for (int i = 0; i < 4; ++i) s.f[i] = 0.f;
#pragma unroll
            for (int j = 0; j < TAPS; ++j) {
                if (j >= p.taps) break;
                const Vec<4>& in = j < halo ? st[n][j < TAPS - 1 ? j : 0] : v;
#pragma unroll
                for (int i = 0; i < 4; ++i) s.f[i] = fmaf(conv[n][j].f[i], in.f[i], s.f[i]);
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) o.f[i] += s.f[i];
#pragma unroll
            for (int j = 0; j < TAPS - 1; ++j) {
                if (j >= halo) break;
                stv<float, 4>(state + (size_t)j * W + c, j + 1 < halo ? st[n][j + 1 < TAPS - 1 ? j + 1 : 0] : v);
            }
        }
        stv<T, 4>(reinterpret_cast<T*>(p.out) + (size_t)row * W + c, o);
    }
}

constexpr int ROWS_THREADS = 512;

// GW warps per row, NV vectors of 4 columns per lane: width <= 128 * GW * NV.  Sixteen warps; blocks, halo rows and state as
// in stack_glue_any_kernel.
template <class T, int GW, int NV>
__global__ void __launch_bounds__(ROWS_THREADS, NV <= 4 ? 2 : 1)
stack_glue_rows_kernel(const __grid_constant__ md_glue p, int R) {
    extern __shared__ __align__(16) float xs[];   // [R + halo][width]
    __shared__ float red[2][ROWS_THREADS / 32];
    constexpr int GROUPS = ROWS_THREADS / 32 / GW;
    const int W = p.width, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int grp = warp / GW, gl = (warp % GW) * 32 + lane;    // this thread's place within its row
    const int t0 = blockIdx.x * R, own = min(R, p.rows - t0), halo = p.conv ? p.taps - 1 : 0;
    const bool first = blockIdx.x == 0;
    md_pdl_launch_dependents();
    // the weights come from HBM once per pass over the model: on their way to L2 before the wait
    for (int i = tid * 32; i < W; i += ROWS_THREADS * 32) {
        prefetch_l2(p.w_pre + i);
        if (p.w_post) prefetch_l2(p.w_post + i);
        for (int j = 0; p.conv && j < p.taps; ++j) prefetch_l2(p.conv + (size_t)j * W + i);
    }
    md_pdl_wait();
    auto total = [&](float v, int turn) {
        v = warp_sum(v);
        if (GW > 1) {
            if (lane == 0) red[turn][warp] = v;
            __syncthreads();
            v = 0.f;
#pragma unroll
            for (int i = 0; i < GW; ++i) v += red[turn][grp * GW + i];
        }
        return v;
    };
    const int slot = halo ? *p.state_slot[0] : 0;
    float* state = halo ? p.state[0] : nullptr;
    if (first && halo)
        for (int i = tid; i < halo * W; i += ROWS_THREADS) xs[i] = state[slot * halo * W + i];
    const int lo = first ? halo : 0, hi = halo + own;      // xs[l] = n[t0 - halo + l]
    for (int l0 = lo; l0 < hi; l0 += GROUPS) {
        const int l = l0 + grp, t = t0 - halo + l;
        const bool live = l < hi;
        Vec<4> x[NV], y[NV];
#pragma unroll
        for (int n = 0; n < NV; ++n) {
#pragma unroll
            for (int i = 0; i < 4; ++i) x[n].f[i] = y[n].f[i] = 0.f;
        }
        const size_t src = live ? (p.gather ? (size_t)p.gather[t] : t) : 0;
        float scale = 1.f;
        if (live) {
            if (p.w_post && !p.slot) {
                const T* yr = reinterpret_cast<const T*>(p.y) + src * W;
#pragma unroll
                for (int n = 0; n < NV; ++n) {
                    const int c = (gl + n * 32 * GW) * 4;
                    if (c < W) y[n] = p.y_f32 ? ldv<float, 4>(p.y_f32 + src * W + c) : ldv<T, 4>(yr + c);
                }
            }
            const T* xe = p.tokens ? reinterpret_cast<const T*>(p.embed) +
                                         (size_t)(p.tokens[src] < (unsigned long long)p.vocab ? p.tokens[src] : 0ull) * W : nullptr;
#pragma unroll
            for (int n = 0; n < NV; ++n) {
                const int c = (gl + n * 32 * GW) * 4;
                if (c < W) x[n] = xe ? ldv<T, 4>(xe + c) : ldv<float, 4>(p.x + src * W + c);
            }
            if (p.w_post && p.ssq) {
                float s = 0.f;
                for (int i = lane; i < p.ssq_parts; i += 32) s += p.ssq[src * p.ssq_parts + i];
                scale = 1.f / sqrtf(warp_sum(s) / (float)p.ssq_n + p.eps);
            }
            if (p.w_post && p.slot)
                for (int k = 0; k < p.top; ++k) {
                    const float s = p.score[src * p.top + k];
                    const T* e = reinterpret_cast<const T*>(p.y) + (size_t)p.slot[src * p.top + k] * W;
#pragma unroll
                    for (int n = 0; n < NV; ++n) {
                        const int c = (gl + n * 32 * GW) * 4;
                        if (c >= W) continue;
                        const Vec<4> v = ldv<T, 4>(e + c);
#pragma unroll
                        for (int i = 0; i < 4; ++i) y[n].f[i] = fmaf(s, v.f[i], y[n].f[i]);
                    }
                }
        }
        if (p.w_post) {
            float ss = 0.f;
#pragma unroll
            for (int n = 0; n < NV; ++n) {
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    y[n].f[i] *= scale;
                    ss = fmaf(y[n].f[i], y[n].f[i], ss);
                }
            }
            const float inv = p.mult / sqrtf(total(ss, 0) / (float)W + p.eps);
#pragma unroll
            for (int n = 0; n < NV; ++n) {
                const int c = (gl + n * 32 * GW) * 4;
                if (c >= W) continue;
                const Vec<4> w = ldv<float, 4>(p.w_post + c);
#pragma unroll
                for (int i = 0; i < 4; ++i) x[n].f[i] = fmaf(y[n].f[i] * inv, w.f[i], x[n].f[i]);
            }
        }
        float ss = 0.f;
        const bool store = live && l >= halo && p.x_out;
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            const int c = (gl + n * 32 * GW) * 4;
#pragma unroll
            for (int i = 0; i < 4; ++i) ss = fmaf(x[n].f[i], x[n].f[i], ss);
            if (store && c < W) stv<float, 4>(p.x_out + (size_t)t * W + c, x[n]);
        }
        const float inv2 = 1.f / sqrtf(total(ss, 1) / (float)W + p.eps);
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            const int c = (gl + n * 32 * GW) * 4;
            if (!live || c >= W) continue;
            const Vec<4> w = ldv<float, 4>(p.w_pre + c);
            Vec<4> v;
#pragma unroll
            for (int i = 0; i < 4; ++i) v.f[i] = x[n].f[i] * (inv2 * w.f[i]);
            stv<float, 4>(xs + (size_t)l * W + c, v);
        }
        if (GW > 1) __syncthreads();    // `red` is free for the next rows
    }
    __syncthreads();
    T* out = reinterpret_cast<T*>(p.out) + (size_t)t0 * W;
    const int per = W / 4;
    for (int i = tid; i < own * per; i += ROWS_THREADS) {
        const int r = i / per, c = (i - r * per) * 4;
        Vec<4> v = lds<4>(xs + (size_t)(r + halo) * W + c);
        if (p.conv) {
            Vec<4> s;
#pragma unroll
            for (int e = 0; e < 4; ++e) s.f[e] = 0.f;
#pragma unroll 4
            for (int j = 0; j < p.taps; ++j) {
                const Vec<4> n = lds<4>(xs + (size_t)(r + j) * W + c), w = ldv<float, 4>(p.conv + (size_t)j * W + c);
#pragma unroll
                for (int e = 0; e < 4; ++e) s.f[e] = fmaf(w.f[e], n.f[e], s.f[e]);
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) v.f[e] += s.f[e];
        }
        stv<T, 4>(out + (size_t)r * W + c, v);
    }
    if (blockIdx.x + 1 < gridDim.x || !halo) return;
    float* dst = state + (size_t)(p.rows == 1 ? slot : slot ^ 1) * halo * W;
    for (int i = tid; i < halo * W; i += ROWS_THREADS) dst[i] = xs[(size_t)own * W + i];
}

// rows of f32 logits -> index of the largest (the lowest index of equal ones)
__global__ void __launch_bounds__(1024)
argmax_f32_kernel(const float* __restrict__ x, size_t n, size_t stride, unsigned long long* __restrict__ out) {
    __shared__ unsigned long long best_s[32];
    md_pdl_launch_dependents();
    md_pdl_wait();
    const float* xr = x + (size_t)blockIdx.x * stride;
    unsigned long long best = 0ull;
    auto take = [&](float v, size_t i) {
        const unsigned long long key = md_argmax_key(v, (uint32_t)i);
        best = key > best ? key : best;
    };
    if ((n % 4) == 0 && ((reinterpret_cast<uintptr_t>(xr)) & 15) == 0) {
        const size_t nv = n / 4;
        for (size_t i0 = threadIdx.x; i0 < nv; i0 += 8 * 1024) {
            float4 v[8];
#pragma unroll
            for (int u = 0; u < 8; ++u)
                if (i0 + u * 1024 < nv) v[u] = __ldcg(reinterpret_cast<const float4*>(xr) + i0 + u * 1024);
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                const size_t i = (i0 + u * 1024) * 4;
                if (i >= n) continue;
                take(v[u].x, i), take(v[u].y, i + 1), take(v[u].z, i + 2), take(v[u].w, i + 3);
            }
        }
    } else {
        for (size_t i = threadIdx.x; i < n; i += blockDim.x) take(xr[i], i);
    }
#pragma unroll
    for (int o = 16; o; o >>= 1) {
        const unsigned long long k = __shfl_xor_sync(0xffffffffu, best, o);
        best = k > best ? k : best;
    }
    if ((threadIdx.x & 31) == 0) best_s[threadIdx.x >> 5] = best;
    __syncthreads();
    if (threadIdx.x == 0) {
        for (unsigned w = 1; w < blockDim.x / 32; ++w) best = best_s[w] > best ? best_s[w] : best;
        out[blockIdx.x] = 0xFFFFFFFFull - (best & 0xFFFFFFFFull);
    }
}

template <class T>
int launch_glue(md_ctx* ctx, const md_glue& g) {
    const int halo = g.conv ? g.taps - 1 : 0;
    const bool v4 = (g.width % 4) == 0;
    const size_t row_bytes = (size_t)g.width * sizeof(float);
    if (g.rows > 1 && g.seqs > 1) return md_fail(ctx, MD_ERR_UNSUPPORTED, "md_glue: several rows of several sequences");
    if (v4 && g.width <= 8192 && g.taps <= 4 && (g.rows == 1 || (g.gather && g.rows <= 8))) {
        const dim3 grid((unsigned)(g.rows * g.seqs));
        if (g.width <= 2048) return md_launch_ex(ctx, stack_glue_step_kernel<T, 1, 4>, grid, dim3(STEP_THREADS), 0, "stack_glue_step_kernel", g);
        if (g.width <= 4096) return md_launch_ex(ctx, stack_glue_step_kernel<T, 2, 4>, grid, dim3(STEP_THREADS), 0, "stack_glue_step_kernel", g);
        return md_launch_ex(ctx, stack_glue_step_kernel<T, 4, 4>, grid, dim3(STEP_THREADS), 0, "stack_glue_step_kernel", g);
    }
    const bool wide = g.rows == 1 || (g.gather && g.rows <= 8);
    int R = wide ? 1 : 8 - halo;
    if (!wide && R < halo) R = halo;
    if (R < 1) R = 1;
    while (!wide && R > halo && R > 1 && (R + halo) * row_bytes > 112 * 1024) --R;   // two blocks per SM where possible
    const size_t smem = (R + halo) * row_bytes;
    if (smem > 220 * 1024) return md_fail(ctx, MD_ERR_UNSUPPORTED, "a width of %d with %d taps exceeds shared memory", g.width, g.taps);
    if (g.x && g.x == g.x_out && g.rows > R) return md_fail(ctx, MD_ERR_INVALID_ARG, "md_glue: in-place residual over several blocks");
    void (*kern)(md_glue, int) = nullptr;
    const bool rows_form = v4 && !wide && g.width <= 16384;
    const unsigned threads = wide ? 512 : rows_form ? ROWS_THREADS : 256;
    if (rows_form)
        kern = g.width <= 512 ? stack_glue_rows_kernel<T, 1, 4> : g.width <= 1024 ? stack_glue_rows_kernel<T, 2, 4>
             : g.width <= 2048 ? stack_glue_rows_kernel<T, 4, 4> : g.width <= 4096 ? stack_glue_rows_kernel<T, 8, 4>
             : g.width <= 8192 ? stack_glue_rows_kernel<T, 16, 4> : stack_glue_rows_kernel<T, 16, 8>;
    else
        kern = wide ? (v4 ? stack_glue_any_kernel<T, 4, true> : stack_glue_any_kernel<T, 1, true>)
                    : (v4 ? stack_glue_any_kernel<T, 4, false> : stack_glue_any_kernel<T, 1, false>);
    if (smem > 47 * 1024) MD_CUDA(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
    return md_launch_ex(ctx, kern, dim3((unsigned)((g.rows + R - 1) / R), (unsigned)g.seqs), dim3(threads), smem,
                        "stack_glue_kernel", g, R);
}

// ---- MD_LAYER_PARALLEL: residual update of two sublayers (the second may be a routed one), one norm, up to two weighted outputs

constexpr int PAR_THREADS = 512;

template <class T> __device__ __forceinline__ const T* embed_row(const md_parallel_glue& p, size_t src) {
    const unsigned long long tok = p.tokens[src];
    return reinterpret_cast<const T*>(p.embed) + (size_t)(tok < (unsigned long long)p.vocab ? tok : 0ull) * p.width;
}
// the first choices of a routed row, requested ahead of everything that does not depend on them
struct Choices { int slot[4]; float score[4]; };
__device__ __forceinline__ Choices first_choices(const md_branch& b, size_t src) {
    Choices c = {};
    if (!b.slot) return c;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
        c.slot[k] = k < b.top ? __ldcg(b.slot + src * b.top + k) : 0;
        c.score[k] = k < b.top ? __ldcg(b.score + src * b.top + k) : 0.f;
    }
    return c;
}
// A thread's vectors (every `step` columns from c0) of a sublayer's output for row `src`, all requested before one is used.
template <class T, int V, int NV>
__device__ __forceinline__ void branch_row(const md_branch& b, const Choices& ch, size_t src, int W, int c0, int step, Vec<V> (&y)[NV]) {
#pragma unroll
    for (int n = 0; n < NV; ++n) {
#pragma unroll
        for (int i = 0; i < V; ++i) y[n].f[i] = 0.f;
    }
    if (b.slot) {
        auto take = [&](int slot, float s) {
            const T* e = reinterpret_cast<const T*>(b.y) + (size_t)slot * W;
#pragma unroll
            for (int n = 0; n < NV; ++n) {
                if (c0 + n * step >= W) continue;
                const Vec<V> v = ldv<T, V>(e + c0 + n * step);
#pragma unroll
                for (int i = 0; i < V; ++i) y[n].f[i] = fmaf(s, v.f[i], y[n].f[i]);
            }
        };
#pragma unroll
        for (int k = 0; k < 4; ++k)
            if (k < b.top) take(ch.slot[k], ch.score[k]);
        for (int k = 4; k < b.top; ++k) take(__ldcg(b.slot + src * b.top + k), __ldcg(b.score + src * b.top + k));
        return;
    }
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        const int c = c0 + n * step;
        if (c >= W) continue;
        y[n] = b.y_f32 ? ldv<float, V>(b.y_f32 + src * W + c) : ldv<T, V>(reinterpret_cast<const T*>(b.y) + src * W + c);
    }
}

// GW warps per row, NV vectors of V columns per lane: width <= 32 * V * GW * NV.  A block walks over rows and keeps its columns'
// weights and scales in registers, requested before the dependency wait.
template <class T, int V, int GW, int NV>
__global__ void __launch_bounds__(PAR_THREADS, NV == 1 ? 2 : 1)
stack_parallel_kernel(const __grid_constant__ md_parallel_glue p) {
    __shared__ float red[2][PAR_THREADS / 32];
    constexpr int GROUPS = PAR_THREADS / 32 / GW;
    const int W = p.width, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int grp = warp / GW, c0 = ((warp % GW) * 32 + lane) * V, step = 32 * GW * V;
    md_pdl_launch_dependents();
    Vec<V> w[2][NV], s[2][NV];
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        const int c = c0 + n * step;
#pragma unroll
        for (int o = 0; o < 2; ++o) {
#pragma unroll
            for (int i = 0; i < V; ++i) w[o][n].f[i] = 0.f, s[o][n].f[i] = 1.f;
            if (c < W && p.out[o]) w[o][n] = ldv<float, V>(p.w[o] + c);
            if (c < W && p.b[o].scale) s[o][n] = ldv<float, V>(p.b[o].scale + c);
        }
    }
    md_pdl_wait();
    int turn = 0;
    for (int row0 = blockIdx.x * GROUPS; row0 < p.rows; row0 += gridDim.x * GROUPS, turn ^= 1) {
        const int row = row0 + grp;
        const bool live = row < p.rows;
        const size_t src = live ? (p.gather ? (size_t)p.gather[row] : row) : 0;
        Vec<V> x[NV];
        const Choices ch = first_choices(p.b[1], src);
        const T* xe = p.tokens ? embed_row<T>(p, src) : nullptr;
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            const int c = c0 + n * step;
#pragma unroll
            for (int i = 0; i < V; ++i) x[n].f[i] = 0.f;
            if (live && c < W) x[n] = xe ? ldv<T, V>(xe + c) : ldv<float, V>(p.x + src * W + c);
        }
#pragma unroll
        for (int b = 0; b < 2; ++b) {
            if ((!p.b[b].y_f32 && !p.b[b].y) || !live) continue;
            Vec<V> y[NV];
            branch_row<T, V, NV>(p.b[b], ch, src, W, c0, step, y);
#pragma unroll
            for (int n = 0; n < NV; ++n) {
#pragma unroll
                for (int i = 0; i < V; ++i) x[n].f[i] = fmaf(s[b][n].f[i], y[n].f[i], x[n].f[i]);
            }
        }
        float ss = 0.f;
#pragma unroll
        for (int n = 0; n < NV; ++n) {
            const int c = c0 + n * step;
#pragma unroll
            for (int i = 0; i < V; ++i) ss = fmaf(x[n].f[i], x[n].f[i], ss);
            if (live && c < W && p.x_out) stv<float, V>(p.x_out + (size_t)row * W + c, x[n]);
        }
        ss = warp_sum(ss);
        if constexpr (GW > 1) {
            if (lane == 0) red[turn][warp] = ss;
            __syncthreads();
            ss = 0.f;
#pragma unroll
            for (int i = 0; i < GW; ++i) ss += red[turn][grp * GW + i];
        }
        const float inv = 1.f / sqrtf(ss / (float)W + p.eps);
#pragma unroll
        for (int o = 0; o < 2; ++o) {
            if (!p.out[o]) continue;
            T* out = reinterpret_cast<T*>(p.out[o]) + (size_t)row * W;
#pragma unroll
            for (int n = 0; n < NV; ++n) {
                const int c = c0 + n * step;
                if (!live || c >= W) continue;
                Vec<V> v;
#pragma unroll
                for (int i = 0; i < V; ++i) v.f[i] = x[n].f[i] * (inv * w[o][n].f[i]);
                stv<T, V>(out + c, v);
            }
        }
    }
}

template <class T, int V>
int launch_parallel_v(md_ctx* ctx, const md_parallel_glue& g) {
    const int per = 32 * V;   // columns a warp holds in one vector per lane
    if (g.width > 128 * per) return md_fail(ctx, MD_ERR_UNSUPPORTED, "a width of %d exceeds %d", g.width, 128 * per);
    const int vectors = (g.width + per - 1) / per;
    void (*kern)(md_parallel_glue) = vectors <= 1 ? stack_parallel_kernel<T, V, 1, 1> : vectors <= 2 ? stack_parallel_kernel<T, V, 2, 1>
                                   : vectors <= 4 ? stack_parallel_kernel<T, V, 4, 1> : vectors <= 8 ? stack_parallel_kernel<T, V, 8, 1>
                                   : vectors <= 16 ? stack_parallel_kernel<T, V, 16, 1> : vectors <= 32 ? stack_parallel_kernel<T, V, 16, 2>
                                   : vectors <= 64 ? stack_parallel_kernel<T, V, 16, 4> : stack_parallel_kernel<T, V, 16, 8>;
    const int groups = vectors <= 1 ? 16 : vectors <= 2 ? 8 : vectors <= 4 ? 4 : vectors <= 8 ? 2 : 1, blocks = (g.rows + groups - 1) / groups;
    const int most = ctx->sm_count * (vectors <= 16 ? 2 : 1);
    return md_launch_ex(ctx, kern, dim3((unsigned)(blocks < most ? blocks : most)), dim3(PAR_THREADS), 0, "stack_parallel_kernel", g);
}

template <class T>
int launch_parallel(md_ctx* ctx, const md_parallel_glue& g) {
    return (g.width % 4) == 0 ? launch_parallel_v<T, 4>(ctx, g) : launch_parallel_v<T, 1>(ctx, g);
}

}  // namespace

int md_launch_glue(md_ctx* ctx, int dtype, const md_glue& g) {
    return dtype == MD_DTYPE_F32 ? launch_glue<float>(ctx, g) : launch_glue<__nv_bfloat16>(ctx, g);
}

int md_launch_parallel_glue(md_ctx* ctx, int dtype, const md_parallel_glue& g) {
    return dtype == MD_DTYPE_F32 ? launch_parallel<float>(ctx, g) : launch_parallel<__nv_bfloat16>(ctx, g);
}

int md_launch_argmax_f32(md_ctx* ctx, const float* x, size_t n, size_t stride, size_t rows, unsigned long long* idx_dev) {
    return md_launch_ex(ctx, argmax_f32_kernel, dim3((unsigned)rows), dim3(1024), 0, "argmax_f32_kernel", x, n, stride, idx_dev);
}
