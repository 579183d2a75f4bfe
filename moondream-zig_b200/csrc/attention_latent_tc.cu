// Latent attention of prompts on the 5th-generation tensor cores (tcgen05 + TMEM + TMA): expanded keys and values, the shared
// rotated key part straight from the cache, sliding window, one sink logit per head (md_latent in stack.cuh).
//
// The division of work is that of attn_tc_kernel (attention_tc.cu): a work item = 128 queries of one head, key tiles of 64, a
// persistent CTA per SM, and per CTA
//   warp 0      TMA producer: an item's Q, K tiles through a ring of three stages, V tiles through a ring of two
//   warp 1      issues S = Q K^T into one of four S buffers in tensor memory;  warp 6 issues O += P V
//   warps 2..5  one thread per query row: its row of Q into tensor memory (the rotated part turned on the way), then per tile its
//               row of S, the softmax, P back over the S buffer.
// What differs: a row of K is two pieces from two tensors, so Q and K travel as 64-dim atoms of the plain part followed by atoms
// of the rotated part (zero filled past either), and the k-steps walk both.  P goes back as two bfloat16 terms, 32 columns each,
// which together fill the S buffer they came from; V is multiplied by both, so the weights keep about 2^-17.  The row sum
// starts at the sink's weight, which is also the first exponent reference: every row has a finite reference from the start.
// Tiles run from the first key of the item's window.  With two S buffers the tile period was the chain PV(j-1) -> S(j+1) ->
// softmax(j+1) (2000 cycles at head sizes 128 + 64, 128); with four it is the longer of the softmax and the products.
//
// Numerics: scores, sums and the output accumulate in f32, one rounding to bfloat16 at the end.  Every mbarrier wait is bounded
// (tc_common.cuh); a wait that gives up is reported through the context's error word and the kernel still runs to its end and
// frees its TMEM.
#include <algorithm>
#include <climits>

#include "stack.cuh"
#include "tc_common.cuh"

int md_make_map_4d(md_ctx* ctx, CUtensorMap* map, const void* ptr, const uint64_t dims[4], const uint64_t strides_bytes[3],
                   uint32_t box0, const uint32_t box_d[3], int swizzle_bytes);

namespace {

using namespace tc;

constexpr int LBQ = 128, LBK = 64, LAT_THREADS = 224;
constexpr int K_STAGES = 3, V_STAGES = 2, MAX_ATOMS = 4, MAX_V_ATOMS = 2;
constexpr uint32_t Q_ATOM = LBQ * 128, K_ATOM = LBK * 128;    // bytes of a 64-dim atom
constexpr uint32_t LAT_TMEM = 512, LT_O = 256, LT_Q = 384;    // four S buffers of 64, O (up to 128), Q (up to 128)
constexpr float LAT_LOG2E = 1.4426950408889634f, LAT_RESCALE = 8.0f;   // see RESCALE_THRESHOLD of attention_tc.cu

struct LatTcParams {
    int rows, pos0, key0, window, heads, n_qblk, n_items;
    int atoms_n, atoms_r, steps_n, steps_r;   // 64-dim atoms and 16-dim k-steps of the plain and of the rotated part
    int vdim, v_cols, rot, negate;            // v_cols: vdim rounded up to 16
    float scale_log2;                         // of the scores' absolute scale; negate: Q changes sign
    const float *sink, *rope;
};
struct LatTcMaps { CUtensorMap qn, qr, kn, kr, v, o; };

struct LatItem { int q0, head, start, nt; };
// Item w: the last query blocks first (they see the most keys).
__device__ __forceinline__ LatItem lat_item(const LatTcParams& p, int w) {
    LatItem i;
    i.q0 = (p.n_qblk - 1 - w / p.heads) * LBQ;
    i.head = w % p.heads;
    i.start = max(0, p.pos0 + i.q0 - p.window + 1);
    i.nt = (p.pos0 + min(i.q0 + LBQ, p.rows) - 1 - i.start) / LBK + 1;
    return i;
}
// The item a CTA takes in its round `it` (-1: none, and none later); rounds alternate direction over the CTAs.
__device__ __forceinline__ int lat_walk(const LatTcParams& p, int it) {
    const int c = (it & 1) ? (int)(gridDim.x - 1 - blockIdx.x) : (int)blockIdx.x;
    const long long w = (long long)it * gridDim.x + c;
    return w < p.n_items ? (int)w : -1;
}

__host__ __device__ constexpr uint32_t lat_smem(int atoms, int v_atoms, int vdim) {
    return 1024 + (uint32_t)atoms * (Q_ATOM + K_STAGES * K_ATOM) + (uint32_t)v_atoms * V_STAGES * K_ATOM + (uint32_t)(LBQ * vdim * 2) + 256;
}

// NV: 64-dim atoms of V
template <int NV>
__global__ void __launch_bounds__(LAT_THREADS, 1)
latent_tc_kernel(const __grid_constant__ LatTcMaps tm, const LatTcParams p, md_devflags* flags) {
    extern __shared__ uint8_t smem_raw[];
    const uint32_t raw = smem_u32(smem_raw), base = (raw + 1023u) & ~1023u;
    uint8_t* base_ptr = smem_raw + (base - raw);
    const uint32_t atoms = (uint32_t)(p.atoms_n + p.atoms_r), q_bytes = atoms * Q_ATOM, k_bytes = atoms * K_ATOM;
    constexpr uint32_t V_BYTES = NV * K_ATOM;
    const uint32_t sm_q = base, sm_k = sm_q + q_bytes, sm_v = sm_k + K_STAGES * k_bytes, sm_out = sm_v + V_STAGES * V_BYTES;
    uint8_t* out_ptr = base_ptr + (sm_out - base);
    const uint32_t bars = sm_out + (uint32_t)(LBQ * p.vdim * 2);
    uint8_t* bars_ptr = base_ptr + (bars - base);
    const uint32_t b_qfull = bars, b_kfull = bars + 8, b_vfull = b_kfull + 8 * K_STAGES;
    const uint32_t b_sfull = b_vfull + 8 * V_STAGES;    // S(j) is in tensor memory: its K stage is free too
    const uint32_t b_pfull = b_sfull + 32;              // the softmax warps have written P(j) over it
    const uint32_t b_pvdone = b_pfull + 32;             // PV(j) has completed: O is current, the S / P buffer and the V stage are free
    const uint32_t b_qcopied = b_pvdone + 32;           // the softmax warps have moved Q from shared to tensor memory
    const uint32_t b_oempty = b_qcopied + 8;            // ... and have read an item's O out of tensor memory
    volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(bars_ptr + 240);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(bars_ptr + 244);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    md_pdl_launch_dependents();
    if (threadIdx.x == 0) {
        tma_prefetch_map(&tm.qn);
        tma_prefetch_map(&tm.qr);
        tma_prefetch_map(&tm.kn);
        tma_prefetch_map(&tm.kr);
        tma_prefetch_map(&tm.v);
        tma_prefetch_map(&tm.o);
        mbar_init(b_qfull, 1);
        mbar_init(b_qcopied, 4);
        mbar_init(b_oempty, 4);
        for (int s = 0; s < K_STAGES; ++s) mbar_init(b_kfull + 8 * s, 1);
        for (int s = 0; s < V_STAGES; ++s) mbar_init(b_vfull + 8 * s, 1);
        for (int b = 0; b < 4; ++b) {
            mbar_init(b_sfull + 8 * b, 1);
            mbar_init(b_pfull + 8 * b, 4);
            mbar_init(b_pvdone + 8 * b, 1);
        }
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(
                         smem_u32(const_cast<uint32_t*>(tmem_slot))),
                     "r"(LAT_TMEM)
                     : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    md_pdl_wait();

    // Every role walks the same items in the same order.  Ring slots, the S / P buffer of a tile and the wait parities run on
    // over the items: `g` counts the key tiles this CTA has handled before the current item.
    if (warp == 0) {
        // ------------------------------------------------------------------ TMA producer
        if (lane == 0) {
            uint32_t kst = 0, vst = 0;       // ring slots
            uint32_t gk = 0, gv = 0;         // K and V tiles loaded so far
            int it = 0;
            for (int w; (w = lat_walk(p, it)) >= 0; ++it) {
                const LatItem i = lat_item(p, w);
                auto load_k = [&](int j) {
                    const int key = i.start + j * LBK;
                    if (gk >= K_STAGES) mbar_wait(b_sfull + 8 * ((gk - K_STAGES) & 3u), ((gk - K_STAGES) >> 2) & 1u, abort_flag, flags, 71);
                    const uint32_t kfull = b_kfull + 8 * kst;
                    uint32_t dst = sm_k + kst * k_bytes;
                    mbar_expect_tx(kfull, k_bytes);
                    for (int a = 0; a < p.atoms_n; ++a, dst += K_ATOM) tma_load_4d(dst, &tm.kn, kfull, a * 64, i.head, key - p.key0, 0);
                    for (int a = 0; a < p.atoms_r; ++a, dst += K_ATOM) tma_load_4d(dst, &tm.kr, kfull, a * 64, key, 0, 0);
                    if (++kst == K_STAGES) kst = 0;
                    ++gk;
                };
                if (it > 0) mbar_wait(b_qcopied, (uint32_t)((it - 1) & 1), abort_flag, flags, 72);
                mbar_expect_tx(b_qfull, q_bytes);
                uint32_t dst = sm_q;
                for (int a = 0; a < p.atoms_n; ++a, dst += Q_ATOM) tma_load_4d(dst, &tm.qn, b_qfull, a * 64, i.head, i.q0, 0);
                for (int a = 0; a < p.atoms_r; ++a, dst += Q_ATOM) tma_load_4d(dst, &tm.qr, b_qfull, a * 64, i.head, i.q0, 0);
                // K runs one tile ahead of V: a K stage comes free with S(j), a V stage only with PV(j)
                load_k(0);
                for (int j = 0; j < i.nt; ++j) {
                    if (j + 1 < i.nt) load_k(j + 1);
                    if (gv >= V_STAGES) mbar_wait(b_pvdone + 8 * ((gv - V_STAGES) & 3u), ((gv - V_STAGES) >> 2) & 1u, abort_flag, flags, 73);
                    const uint32_t vfull = b_vfull + 8 * vst, vdst = sm_v + vst * V_BYTES;
                    mbar_expect_tx(vfull, V_BYTES);
#pragma unroll
                    for (int a = 0; a < NV; ++a) tma_load_4d(vdst + a * K_ATOM, &tm.v, vfull, a * 64, i.head, i.start + j * LBK - p.key0, 0);
                    if (++vst == V_STAGES) vst = 0;
                    ++gv;
                }
            }
            if (*abort_flag) {  // let copies in flight land before the CTA's shared memory is released
                const unsigned long long t0 = global_ns();
                while (global_ns() - t0 < 500000ull) {}
            }
        }
    } else if (warp == 1) {
        // ------------------------------------------------------------------ issuer of the S products
        if (lane == 0) {
            const uint32_t idesc_s = idesc_format<true>() | (1u << 4) | ((uint32_t)(LBK >> 3) << 17) | ((uint32_t)(LBQ >> 4) << 24);
            const uint32_t hi128 = desc_hi(1024, 2), k_lo0 = desc_lo(sm_k, 16), stage16 = k_bytes >> 4;
            uint32_t st = 0, par = 0;        // ring slot and parity of the next S product
            uint32_t g = 0;                  // key tiles of earlier items
            int it = 0;
            for (int w; (w = lat_walk(p, it)) >= 0; ++it) {
                const int nt = lat_item(p, w).nt;
                mbar_wait(b_qcopied, (uint32_t)(it & 1), abort_flag, flags, 74);
                for (int j = 0; j < nt; ++j) {
                    const uint32_t gj = g + (uint32_t)j, sb = gj & 3u;
                    mbar_wait(b_kfull + 8 * st, par, abort_flag, flags, 75);
                    // the buffer still holds P of four tiles back until that PV product has completed
                    mbar_wait(b_pvdone + 8 * sb, ((gj >> 2) & 1u) ^ 1u, abort_flag, flags, 76);
                    tc_fence_after();
                    const uint32_t t_s = tmem_base + sb * 64u;
                    // a k-step of 16 dims: 8 columns of Q, 32 bytes within an atom of K.  What the issuing thread does between
                    // two MMAs is tensor-pipe idle time, so whole atoms are unrolled.
                    uint32_t k_lo = k_lo0 + st * stage16, t_q = tmem_base + LT_Q;
                    tc_mma_f16_ts<false>(t_s, t_q, k_lo, hi128, idesc_s);
                    int skip = 1;
                    auto part = [&](int steps) {
                        for (; steps > 0; steps -= 4, k_lo += K_ATOM >> 4, t_q += 32, skip = 0) {
                            if (!skip) tc_mma_f16_ts<true>(t_s, t_q, k_lo, hi128, idesc_s);
                            if (steps >= 4) {
#pragma unroll
                                for (int ks = 1; ks < 4; ++ks) tc_mma_f16_ts<true>(t_s, t_q + ks * 8, k_lo + ks * 2, hi128, idesc_s);
                            } else {
                                for (int ks = 1; ks < steps; ++ks) tc_mma_f16_ts<true>(t_s, t_q + ks * 8, k_lo + ks * 2, hi128, idesc_s);
                            }
                        }
                    };
                    part(p.steps_n);
                    part(p.steps_r);
                    tc_commit(b_sfull + 8 * sb);
                    if (++st == K_STAGES) { st = 0; par ^= 1u; }
                }
                g += (uint32_t)nt;
            }
        }
    } else if (warp == 6) {
        // ------------------------------------------------------------------ issuer of the PV products
        if (lane == 0) {
            const uint32_t idesc_pv =
                idesc_format<true>() | (1u << 4) | (1u << 16) | ((uint32_t)(p.v_cols >> 3) << 17) | ((uint32_t)(LBQ >> 4) << 24);
            // V: MN-major, 64 dims contiguous per key; the next atom along the dims lies K_ATOM further
            const uint32_t hi128 = desc_hi(1024, 2), v_lo0 = desc_lo(sm_v, K_ATOM);
            uint32_t st = 0, par = 0;        // ring slot and parity of the next PV product
            uint32_t g = 0;
            int it = 0;
            for (int w; (w = lat_walk(p, it)) >= 0; ++it) {
                const int nt = lat_item(p, w).nt;
                for (int j = 0; j < nt; ++j) {
                    const uint32_t gj = g + (uint32_t)j, pb = gj & 3u;
                    mbar_wait(b_vfull + 8 * st, par, abort_flag, flags, 77);
                    mbar_wait(b_pfull + 8 * pb, (gj >> 2) & 1u, abort_flag, flags, 78);
                    // the first product of an item overwrites O: the previous item's output must have left tensor memory
                    if (j == 0 && it > 0) mbar_wait(b_oempty, (uint32_t)((it - 1) & 1), abort_flag, flags, 79);
                    tc_fence_after();
                    const uint32_t t_p = tmem_base + pb * 64u, v_lo = v_lo0 + st * (V_BYTES >> 4);
                    // 16 keys = 8 columns of P and 2048 B of V per k-step (in every atom); both terms of P against the same V
                    if (j == 0) tc_mma_f16_ts<false>(tmem_base + LT_O, t_p, v_lo, hi128, idesc_pv);
                    else tc_mma_f16_ts<true>(tmem_base + LT_O, t_p, v_lo, hi128, idesc_pv);
                    tc_mma_f16_ts<true>(tmem_base + LT_O, t_p + 32, v_lo, hi128, idesc_pv);
#pragma unroll
                    for (int ks = 1; ks < LBK / 16; ++ks) {
                        tc_mma_f16_ts<true>(tmem_base + LT_O, t_p + ks * 8, v_lo + ks * 128, hi128, idesc_pv);
                        tc_mma_f16_ts<true>(tmem_base + LT_O, t_p + 32 + ks * 8, v_lo + ks * 128, hi128, idesc_pv);
                    }
                    tc_commit(b_pvdone + 8 * pb);
                    if (++st == V_STAGES) { st = 0; par ^= 1u; }
                }
                g += (uint32_t)nt;
            }
        }
    } else {
        // ------------------------------------------------------------------ softmax + output (warps 2..5)
        const int quad = warp & 3, row = quad * 32 + lane;
        const uint32_t t_lane = tmem_base + ((uint32_t)(quad * 32) << 16);
        const uint32_t sign = p.negate ? 0x80008000u : 0u;
        const int out_row = p.vdim * 2;
        uint8_t* stage_row = out_ptr + row * out_row;                            // this row in the output staging
        const uint32_t stage_warp = sm_out + (uint32_t)(quad * 32 * out_row);    // this warp's 32 rows of it
        // This row of Q of the CTA's item number `item`: out of the swizzled atoms (16-byte chunk c of a 128-byte row sits at
        // c ^ (row & 7)) into tensor memory, two dims per column; the rotated part is turned by the row's position.  Called once
        // every S product of the item before has completed (its last PV product was waited for).
        auto copy_q = [&](int item, int q0) {
            mbar_wait(b_qfull, (uint32_t)(item & 1), abort_flag, flags, 80);
            const float4* cs = reinterpret_cast<const float4*>(p.rope + (size_t)(p.pos0 + min(q0 + row, p.rows - 1)) * p.rot);
            for (int a = 0; a < (int)atoms; ++a) {
                const uint8_t* q_row = base_ptr + a * Q_ATOM + row * 128;
                uint32_t col = t_lane + LT_Q + (uint32_t)a * 32u;
#pragma unroll
                for (int h = 0; h < 2; ++h) {
                    uint32_t qa[16];
#pragma unroll
                    for (int c = 0; c < 4; ++c) {
                        const uint4 v = *reinterpret_cast<const uint4*>(q_row + (((4 * h + c) ^ (row & 7)) << 4));
                        qa[4 * c] = v.x; qa[4 * c + 1] = v.y; qa[4 * c + 2] = v.z; qa[4 * c + 3] = v.w;
                    }
                    if (a >= p.atoms_n) {
                        const int pair0 = (a - p.atoms_n) * 32 + h * 16;     // rotated pairs pair0 .. + 15, two per float4
#pragma unroll
                        for (int e = 0; e < 16; e += 2) {
                            if (pair0 + e < p.rot / 2) {
                                const float4 c = __ldg(cs + (pair0 + e) / 2);
#pragma unroll
                                for (int k = 0; k < 2; ++k) {
                                    const float u = __uint_as_float(qa[e + k] << 16), v = __uint_as_float(qa[e + k] & 0xffff0000u);
                                    const float co = k ? c.z : c.x, si = k ? c.w : c.y;
                                    qa[e + k] = md_pack_bf16(u * co - v * si, v * co + u * si);
                                }
                            }
                        }
                    }
#pragma unroll
                    for (int e = 0; e < 16; ++e) qa[e] ^= sign;
                    tc_st_32x16(col + 16 * h, qa);
                }
            }
            tc_wait_st();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(b_qcopied);
        };
        uint32_t g = 0;
        int it = 0;
        if (lat_walk(p, 0) >= 0) copy_q(0, lat_item(p, lat_walk(p, 0)).q0);
        for (int w; (w = lat_walk(p, it)) >= 0; ++it) {
            const LatItem i = lat_item(p, w);
            const int nt = i.nt, qpos = p.pos0 + i.q0 + row, wpos = p.pos0 + i.q0 + quad * 32;
            const bool row_ok = i.q0 + row < p.rows;
            // exponent reference (log2 units) and row sum on that reference: the sink's weight to begin with
            float m_run = p.sink[i.head] * LAT_LOG2E, l_run = 1.f;

            for (int j = 0; j < nt; ++j) {
                const uint32_t gj = g + (uint32_t)j;
                const int sb = (int)(gj & 3u), k0 = i.start + j * LBK;
                mbar_wait(b_sfull + 8 * sb, (gj >> 2) & 1u, abort_flag, flags, 81);
                tc_fence_after();
                uint32_t s0[32], s1[32];
                tc_ld_32x32(t_lane + (uint32_t)(sb * 64), s0);
                tc_ld_32x32(t_lane + (uint32_t)(sb * 64 + 32), s1);
                tc_wait_ld();
                // the visible keys of a row are a run of the tile: from n_lo up to n_hi (all of them in most tiles)
                if (!(k0 + LBK - 1 <= wpos && wpos + 31 - k0 < p.window && i.q0 + quad * 32 + 31 < p.rows)) {
                    const int n_hi = row_ok ? qpos - k0 + 1 : 0, n_lo = qpos - p.window + 1 - k0;
#pragma unroll
                    for (int e = 0; e < 32; ++e) {
                        if (e >= n_hi || e < n_lo) s0[e] = 0xff800000u;  // -inf
                        if (e + 32 >= n_hi || e + 32 < n_lo) s1[e] = 0xff800000u;
                    }
                }
                // three-input max (two new values per instruction), eight independent chains of four
                float mx[8];
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    mx[c] = fmaxf(__uint_as_float(s0[8 * c]), __uint_as_float(s0[8 * c + 1]));
                    mx[4 + c] = fmaxf(__uint_as_float(s1[8 * c]), __uint_as_float(s1[8 * c + 1]));
                }
#pragma unroll
                for (int e = 2; e < 8; e += 2) {
#pragma unroll
                    for (int c = 0; c < 4; ++c) {
                        mx[c] = max3(mx[c], __uint_as_float(s0[8 * c + e]), __uint_as_float(s0[8 * c + e + 1]));
                        mx[4 + c] = max3(mx[4 + c], __uint_as_float(s1[8 * c + e]), __uint_as_float(s1[8 * c + e + 1]));
                    }
                }
                const float mt = fmaxf(max3(mx[0], mx[1], mx[2]), max3(max3(mx[3], mx[4], mx[5]), mx[6], mx[7])) * p.scale_log2;
                if (j == 0) {
                    const float m_new = fmaxf(m_run, mt);
                    l_run = ex2_fast(m_run - m_new);
                    m_run = m_new;
                } else if (__any_sync(0xffffffffu, mt > m_run + LAT_RESCALE)) {
                    // move this warp's rows to their new maxima: O(row) *= 2^(old - new), once PV(j-1) has landed
                    const float m_new = fmaxf(m_run, mt), corr = ex2_fast(m_run - m_new);
                    l_run *= corr;
                    m_run = m_new;
                    mbar_wait(b_pvdone + 8 * ((gj - 1) & 3u), ((gj - 1) >> 2) & 1u, abort_flag, flags, 82);
                    tc_fence_after();
#pragma unroll
                    for (int c = 0; c < NV * 4; ++c) {
                        if (c * 16 >= p.v_cols) break;
                        uint32_t r[16];
                        tc_ld_32x16(t_lane + LT_O + c * 16, r);
                        tc_wait_ld();
#pragma unroll
                        for (int e = 0; e < 16; ++e) r[e] = __float_as_uint(__uint_as_float(r[e]) * corr);
                        tc_st_32x16(t_lane + LT_O + c * 16, r);
                    }
                }
                const float neg_m = -m_run;
                float rs[8];   // eight independent partial sums
#pragma unroll
                for (int c = 0; c < 8; ++c) rs[c] = 0.f;
                // P over the S buffer it came from (this thread has its whole S row in registers): column c holds keys 2c, 2c + 1;
                // first terms in the first 32 columns, second terms in the others
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    uint32_t hi[16], lo[16];
#pragma unroll
                    for (int e = 0; e < 16; ++e) {
                        const uint32_t x0 = half ? s1[2 * e] : s0[2 * e], x1 = half ? s1[2 * e + 1] : s0[2 * e + 1];
                        const float a0 = ex2_fast(fmaf(__uint_as_float(x0), p.scale_log2, neg_m));
                        const float a1 = ex2_fast(fmaf(__uint_as_float(x1), p.scale_log2, neg_m));
                        rs[(e & 3) * 2] += a0; rs[(e & 3) * 2 + 1] += a1;
                        hi[e] = md_pack_bf16(a0, a1);
                        lo[e] = md_pack_bf16(a0 - __uint_as_float(hi[e] << 16), a1 - __uint_as_float(hi[e] & 0xffff0000u));
                    }
                    tc_st_32x16(t_lane + (uint32_t)(sb * 64 + 16 * half), hi);
                    tc_st_32x16(t_lane + (uint32_t)(sb * 64 + 32 + 16 * half), lo);
                }
                l_run += ((rs[0] + rs[1]) + (rs[2] + rs[3])) + ((rs[4] + rs[5]) + (rs[6] + rs[7]));
                tc_wait_st();
                tc_fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(b_pfull + 8 * sb);
            }

            // The item's output: out of tensor memory into registers first.  That frees O, and with it the next item can start:
            // its Q goes into tensor memory now, so its first S product runs while this item's output is converted and stored.
            uint32_t o[NV * 4][16];
            const uint32_t gl = g + (uint32_t)nt - 1u;
            mbar_wait(b_pvdone + 8 * (gl & 3u), (gl >> 2) & 1u, abort_flag, flags, 83);
            tc_fence_after();
#pragma unroll
            for (int c = 0; c < NV * 4; ++c) {
                if (c * 16 >= p.v_cols) break;
                tc_ld_32x16(t_lane + LT_O + c * 16, o[c]);
            }
            tc_wait_ld();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(b_oempty);
            if (lat_walk(p, it + 1) >= 0) copy_q(it + 1, lat_item(p, lat_walk(p, it + 1)).q0);

            // the warp's 32 rows are packed in shared memory and leave as one TMA store (rows past the end are clipped by the map)
            if (lane == 0) tma_store_wait_read<0>();   // the previous item's store has read the staging rows
            __syncwarp();
            const float inv = 1.0f / l_run;
#pragma unroll
            for (int c = 0; c < NV * 4; ++c) {
#pragma unroll
                for (int h8 = 0; h8 < 2; ++h8) {
                    if (c * 16 + h8 * 8 < p.vdim) {
                        uint32_t wv[4];
#pragma unroll
                        for (int e = 0; e < 4; ++e)
                            wv[e] = md_pack_bf16(__uint_as_float(o[c][h8 * 8 + 2 * e]) * inv, __uint_as_float(o[c][h8 * 8 + 2 * e + 1]) * inv);
                        *reinterpret_cast<uint4*>(stage_row + (c * 16 + h8 * 8) * 2) = make_uint4(wv[0], wv[1], wv[2], wv[3]);
                    }
                }
            }
            fence_async_smem();
            __syncwarp();
            if (lane == 0 && i.q0 + quad * 32 < p.rows) {
                tma_store_4d(&tm.o, stage_warp, 0, i.head, i.q0 + quad * 32, 0);
                tma_store_commit();
            }
            g += (uint32_t)nt;
        }
        if (lane == 0) tma_store_wait_all();
    }

    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(LAT_TMEM) : "memory");
    }
}

// (dim, head, row) map of `heads` x `rows` vectors of `d` values, boxes of `box_d` values of `box_rows` rows of one head
int vector_map(md_ctx* ctx, CUtensorMap* map, const void* ptr, size_t d, size_t heads, size_t rows, size_t head_stride, size_t row_stride,
               uint32_t box_d, uint32_t box_rows, int swizzle) {
    const uint64_t dims[4] = {d, heads, rows, 1}, strides[3] = {head_stride * 2, row_stride * 2, row_stride * rows * 2};
    const uint32_t box[3] = {1, box_rows, 1};
    return md_make_map_4d(ctx, map, ptr, dims, strides, box_d, box, swizzle);
}

}  // namespace

bool md_latent_tc_supported(const md_latent& a) {
    const int atoms = (a.dim + 63) / 64 + (a.rot + 63) / 64;
    const uintptr_t ptrs = reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(a.kv) | reinterpret_cast<uintptr_t>(a.kr[0]) |
                           reinterpret_cast<uintptr_t>(a.out);
    return atoms <= MAX_ATOMS && a.vdim <= 64 * MAX_V_ATOMS && (a.dim % 8) == 0 && (a.rot % 8) == 0 && (a.vdim % 8) == 0 && (ptrs & 15) == 0;
}

// Keys key0 .. pos0 + rows are expanded in a.kv.
int md_launch_latent_tc(md_ctx* ctx, const md_latent& a, int key0) {
    if (!md_latent_tc_supported(a)) return md_fail(ctx, MD_ERR_UNSUPPORTED, "tcgen05 latent attention: head sizes %d + %d, %d", a.dim, a.rot, a.vdim);
    typedef const uint16_t* half_ptr;
    const size_t D = a.dim, rot = a.rot, E = a.vdim, H = a.heads, per_q = H * (D + rot), per_kv = H * (D + E);
    const size_t keys = (size_t)a.pos0 + a.rows - key0;
    LatTcMaps tm;
    half_ptr q = reinterpret_cast<half_ptr>(a.q), kv = reinterpret_cast<half_ptr>(a.kv);
    MD_TRY(vector_map(ctx, &tm.qn, q, D, H, a.rows, D + rot, per_q, 64, LBQ, 128));
    MD_TRY(vector_map(ctx, &tm.kn, kv, D, H, keys, D, per_kv, 64, LBK, 128));
    MD_TRY(vector_map(ctx, &tm.v, kv + H * D, E, H, keys, E, per_kv, 64, LBK, 128));
    MD_TRY(vector_map(ctx, &tm.o, a.out, E, H, a.rows, E, H * E, (uint32_t)E, 32, 0));
    tm.qr = tm.qn, tm.kr = tm.kn;
    if (rot) {
        MD_TRY(vector_map(ctx, &tm.qr, q + D, rot, H, a.rows, D + rot, per_q, 64, LBQ, 128));
        // rows of one vector each: (dim, row)
        const uint64_t dims[4] = {rot, (uint64_t)a.pos0 + a.rows, 1, 1}, bytes = rot * 2, all = bytes * ((uint64_t)a.pos0 + a.rows);
        const uint64_t strides[3] = {bytes, all, all};
        const uint32_t box[3] = {LBK, 1, 1};
        MD_TRY(md_make_map_4d(ctx, &tm.kr, a.kr[0], dims, strides, 64, box, 128));
    }
    LatTcParams p = {};
    p.rows = a.rows, p.pos0 = a.pos0, p.key0 = key0, p.window = a.window > 0 ? a.window : 0x3fffffff, p.heads = a.heads;
    p.n_qblk = (a.rows + LBQ - 1) / LBQ;
    const size_t items = (size_t)p.n_qblk * H;
    if (items > (size_t)INT_MAX) return md_fail(ctx, MD_ERR_UNSUPPORTED, "tcgen05 latent attention: too many query blocks");
    p.n_items = (int)items;
    p.atoms_n = (a.dim + 63) / 64, p.atoms_r = (a.rot + 63) / 64, p.steps_n = (a.dim + 15) / 16, p.steps_r = (a.rot + 15) / 16;
    p.vdim = a.vdim, p.v_cols = (a.vdim + 15) / 16 * 16, p.rot = a.rot, p.negate = a.scale < 0.f;
    p.scale_log2 = std::max(fabsf(a.scale) * LAT_LOG2E, 1e-30f);
    p.sink = a.sink, p.rope = a.rope;
    const int nv = (a.vdim + 63) / 64;
    const uint32_t smem = lat_smem(p.atoms_n + p.atoms_r, nv, a.vdim);
    auto kern = nv == 1 ? latent_tc_kernel<1> : latent_tc_kernel<2>;
    MD_CUDA(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    return md_launch_ex(ctx, kern, dim3((unsigned)std::min(items, (size_t)ctx->sm_count)), dim3(LAT_THREADS), smem, "latent_tc_kernel", tm, p,
                        ctx->flags);
}
