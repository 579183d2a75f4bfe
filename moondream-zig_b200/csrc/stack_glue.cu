// What sits between the matrix products of a layer-stack decoder: residual update, RMS norms and the causal
// convolution in one kernel (md_glue in stack.cuh states the arithmetic), the append of new keys to a cache, and the
// greedy sample of f32 logits.  Everything is f32; only the row handed to the next product is rounded to T.
#include "stack.cuh"

namespace {

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

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
// of them; the first block of a sequence takes those from the state instead, and is the only one that touches the state:
// it reads the old one before it recomputes the sequence's last taps - 1 rows and stores them.
template <class T, int V, bool WIDE>
__global__ void __launch_bounds__(WIDE ? 512 : 256)
stack_glue_kernel(const __grid_constant__ md_glue p, int R) {
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

    float* state = halo ? p.state[seq] : nullptr;
    if (first && halo)
        for (int i = tid; i < halo * W; i += blockDim.x) xs[i] = state[i];
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
    if (!first || !halo) return;
    // the sequence's last taps - 1 values of n: in xs if this block holds the whole sequence (older ones are the old
    // state, which sits in xs[0 .. halo) ), otherwise recomputed
    int base = p.rows;
    if (p.rows > own) {
        __syncthreads();
        if (WIDE) {
            for (int l = 0; l < halo; ++l) row(l, p.rows - halo + l, false);
        } else {
            for (int l = warp; l < halo; l += 8) row(l, p.rows - halo + l, false);
        }
        base = 0;
        __syncthreads();
    }
    for (int i = tid; i < halo * W; i += blockDim.x) state[i] = xs[(size_t)base * W + i];
}

// rows of f32 logits -> index of the largest (the lowest index of equal ones)
__global__ void __launch_bounds__(1024)
argmax_f32_kernel(const float* __restrict__ x, size_t n, size_t stride, unsigned long long* __restrict__ out) {
    __shared__ unsigned long long best_s[32];
    md_pdl_launch_dependents();
    md_pdl_wait();
    const float* xr = x + (size_t)blockIdx.x * stride;
    unsigned long long best = 0ull;   // (order-preserving image of the value) << 32 | ~index
    for (size_t i = threadIdx.x; i < n; i += blockDim.x) {
        const uint32_t b = __float_as_uint(xr[i]);
        const uint32_t o = (b & 0x80000000u) ? ~b : (b | 0x80000000u);
        const unsigned long long key = ((unsigned long long)o << 32) | (0xFFFFFFFFull - i);
        best = key > best ? key : best;
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
    const bool wide = g.rows == 1 || (g.gather && g.rows <= 8);
    const size_t row_bytes = (size_t)g.width * sizeof(float);
    int R = wide ? 1 : 8 - halo;
    if (!wide && R < halo) R = halo;
    if (R < 1) R = 1;
    while (!wide && R > halo && R > 1 && (R + halo) * row_bytes > 100 * 1024) --R;   // two blocks per SM where possible
    const size_t smem = (R + halo) * row_bytes;
    if (smem > 220 * 1024) return md_fail(ctx, MD_ERR_UNSUPPORTED, "a width of %d with %d taps exceeds shared memory", g.width, g.taps);
    if (g.x && g.x == g.x_out && g.rows > R) return md_fail(ctx, MD_ERR_INVALID_ARG, "md_glue: in-place residual over several blocks");
    const bool v4 = (g.width % 4) == 0;
    auto kern = wide ? (v4 ? stack_glue_kernel<T, 4, true> : stack_glue_kernel<T, 1, true>)
                     : (v4 ? stack_glue_kernel<T, 4, false> : stack_glue_kernel<T, 1, false>);
    if (smem > 47 * 1024) MD_CUDA(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
    return md_launch_ex(ctx, kern, dim3((unsigned)((g.rows + R - 1) / R), (unsigned)g.seqs), dim3(wide ? 512 : 256), smem,
                        "stack_glue_kernel", g, R);
}

}  // namespace

int md_launch_glue(md_ctx* ctx, int dtype, const md_glue& g) {
    return dtype == MD_DTYPE_F32 ? launch_glue<float>(ctx, g) : launch_glue<__nv_bfloat16>(ctx, g);
}

int md_launch_argmax_f32(md_ctx* ctx, const float* x, size_t n, size_t stride, size_t rows, unsigned long long* idx_dev) {
    return md_launch_ex(ctx, argmax_f32_kernel, dim3((unsigned)rows), dim3(1024), 0, "argmax_f32_kernel", x, n, stride, idx_dev);
}
