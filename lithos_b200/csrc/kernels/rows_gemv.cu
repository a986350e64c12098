// Dense bf16 rows x one fp32 vector for the decode step of bf16 models: one launch takes one or two matrices, builds the input
// vector(s) in shared memory (RMS norm with the layer's weights; or the mixer's output with its per-head norm and gate, followed
// by the feed-forward's activations) and finishes every row (store, gated product of neighbouring rows, squared ReLU, residual add, soft cap
// with arg-max candidates).  A matrix may be a stack of experts of which the token uses a few: their rows, or their columns, follow one another.  The vector stays fp32; weights are exact in fp32, sums are fp32 in a fixed order.
//
// HBM-bound: one CTA per SM, every warp streams its own row segments with 1-D bulk copies through its own ring, so what is in flight
// (ring bytes x 148) does not depend on registers.  Two rows share every read of the vector: shared memory moves 2 bytes of weights in,
// 2 out and 2 bytes of vector per weight.  Narrow launches (fewer pairs than warps per CTA) cut a pair into segments, one per warp turn;
// the segments of a pair are added in order, so a result does not depend on the schedule.  Where the vector is so long that it would leave
// the ring too shallow, two CTAs (a cluster) take half of K each: half the vector to gather and to hold, and the sums of the two halves are
// added, in order, through distributed shared memory.
#include "common.cuh"
#include "params.h"

__device__ __forceinline__ void rg_cluster_sync() {
    asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ float2 rg_ld_cluster(const float* local_ptr, uint32_t rank) {
    uint32_t remote;
    float2 v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(smem_u32(local_ptr)), "r"(rank));
    asm volatile("ld.shared::cluster.v2.f32 {%0, %1}, [%2];" : "=f"(v.x), "=f"(v.y) : "r"(remote) : "memory");
    return v;
}
__device__ __forceinline__ float rg_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }

// NORM: the norm of LB_RG_X_NORM; SEL: matrices are stacks of experts
template <int NORM, bool SEL>
__device__ __forceinline__ void rows_gemv_body(const lb_rows_gemv_params& p) {
    extern __shared__ __align__(16) unsigned char rg_sm[];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int G = gridDim.x, c = blockIdx.x, S = p.stages;
    // gridDim.y = 2 (a cluster along y): this CTA's half of the row segments, columns k_lo .. k_hi - 1
    const int KS = gridDim.y, rank = blockIdx.y, seg_lo = rank * p.segs / KS, my_segs = (rank + 1) * p.segs / KS - seg_lo;
    const int k_lo = seg_lo * LB_RG_SEG, k_hi = min(p.K, k_lo + my_segs * LB_RG_SEG);
    const int split = p.split > 1 ? my_segs : 1, spp = p.split > 1 ? 1 : my_segs; // pieces of a row pair, segments of a piece
    const int pairs0 = (p.mat[0].rows + 1) >> 1, pairs1 = p.n_mat > 1 ? (p.mat[1].rows + 1) >> 1 : 0, P = pairs0 + pairs1;
    const int my_pairs = P > c ? (P - c + G - 1) / G : 0;
    const int n_vec = p.x_mode == LB_RG_X_NORM ? p.n_mat : 1;
    unsigned char* ring = rg_sm;                                                              // [warps][S][2][SEG] bf16
    float* xsm = reinterpret_cast<float*>(ring + (size_t)LB_RG_WARPS * S * LB_RG_SEG * 4);     // [n_vec][K] (its half)
    float* gate_s = xsm + (size_t)n_vec * p.x_cols;                                                // [n_mix] when there is a gate
    float* part = gate_s + (p.gate ? (p.n_mix + 3) & ~3 : 0);                                  // [my_pairs * split][2]
    const int max_pairs = (P + G - 1) / G;
    float* red = part + (size_t)2 * max_pairs * p.split;                                      // [40]
    uint64_t* bars = reinterpret_cast<uint64_t*>(red + 40);                                    // [warps][S], the vector's
    if (lane == 0)
        for (int s = 0; s < S; ++s) mbar_init(&bars[warp * S + s], 1);
    if (tid == 0) mbar_init(&bars[LB_RG_WARPS * S], 1);
    mbar_fence_init();
    __shared__ int sel_s[LB_RG_MAX_PARTS];
    if (SEL && tid < p.parts) sel_s[tid] = p.sel[(size_t)p.sel_row[0] * p.parts + tid];
    __syncthreads();

    // the warp's stages: items warp, warp + 8, ... (item = pair * split + piece), segments of the item in order
    const int items = my_pairs * split;
    const uint64_t pol = l2_policy_evict_first();
    auto row_ptr = [&](int pair, int& mi) -> const uint16_t* {
        const int g = c + pair * G;
        mi = g >= pairs0;
        if (SEL && p.x_mode == LB_RG_X_NORM) { // the parts' rows one after the other, each part's from its expert
            const int part_pairs = p.sel_rows >> 1, e = g / part_pairs;
            return p.mat[0].w + ((size_t)sel_s[e] * part_pairs + (g - e * part_pairs)) * 2 * p.K;
        }
        return mi ? p.mat[1].w + (size_t)(g - pairs0) * 2 * p.K : p.mat[0].w + (size_t)g * 2 * p.K;
    };
    // a row segment: its first column and length; with experts side by side along K a row is in pieces of k_part columns
    const bool sel_k = SEL && p.x_mode == LB_RG_X_CAT;
    const size_t row_step = sel_k ? p.k_part : p.K, expert_pairs = sel_k ? (size_t)((p.mat[0].rows + 1) >> 1) : 0;
    auto segment = [&](int seg, int& col, int& len, int& e) {
        if (SEL && sel_k) {
            e = seg / p.segs_part;
            const int off = (seg - e * p.segs_part) * LB_RG_SEG;
            col = e * p.k_part + off;
            len = min(LB_RG_SEG, p.k_part - off);
        } else {
            col = seg * LB_RG_SEG;
            len = min(LB_RG_SEG, p.K - col);
        }
    };
    int r_item = warp, r_seg = 0, r_slot = 0; // next stage to request
    auto request = [&]() {
        if (r_item >= items) return;
        if (lane == 0) {
            const int pair = split == 1 ? r_item : r_item / split, seg = seg_lo + (r_item - pair * split) * spp + r_seg;
            int mi, col, len, e = 0;
            segment(seg, col, len, e);
            const uint16_t* w = SEL && sel_k ? p.mat[0].w + ((size_t)sel_s[e] * expert_pairs + (c + pair * G)) * 2 * p.k_part + (col - e * p.k_part) : row_ptr(pair, mi) + col;
            const uint32_t bytes = (uint32_t)len * 2u;
            unsigned char* dst = ring + (size_t)(warp * S + r_slot) * (LB_RG_SEG * 4);
            uint64_t* bar = &bars[warp * S + r_slot];
            mbar_arrive_expect_tx(bar, 2 * bytes);
            bulk_g2s(dst, w, bytes, bar, pol);
            bulk_g2s(dst + LB_RG_SEG * 2, w + row_step, bytes, bar, pol);
        }
        if (++r_seg == spp) { r_seg = 0; r_item += LB_RG_WARPS; }
        if (++r_slot == S) r_slot = 0;
    };
    for (int s = 0; s < S; ++s) request(); // weights are constants: asked for before the previous kernel has finished

    // the norm weights are constants too: a thread's first 8 quads of them (of the two vectors, or weight and bias of one) come in before
    // the wait
    constexpr bool layer_norm = NORM == LB_NORM_LAYER;
    const uint16_t* second = n_vec > 1 ? p.mat[1].norm_w : layer_norm ? p.mat[0].norm_b : nullptr;
    const bool quads = (p.width & 3) == 0;
    uint2 w_pre[2][8];
    if (p.x_mode == LB_RG_X_NORM && quads) {
#pragma unroll
        for (int v = 0; v < 2; ++v)
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                const int i = 4 * (tid + u * LB_RG_THREADS);
                const uint16_t* src = v == 0 ? p.mat[0].norm_w : second;
                w_pre[v][u] = src && i < p.width ? __ldg(reinterpret_cast<const uint2*>(src + i)) : make_uint2(0u, 0u);
            }
    }
    // the vector's parts come as bulk copies straight into its place (whole 16-byte pieces; what is left over by plain loads), so the
    // launch waits for one trip to L2 and not for as many as a thread has loads in turn
    uint64_t* xbar = bars + LB_RG_WARPS * S;
    pdl_wait();
    if (p.x_mode == LB_RG_X_NORM) {
        const int n4 = p.width & ~3;
        if (tid == 0) {
            mbar_arrive_expect_tx(xbar, (uint32_t)n4 * 4u);
            if (n4) bulk_g2s_plain(xsm, p.x, (uint32_t)n4 * 4u, xbar);
        }
        for (int i = n4 + tid; i < p.width; i += LB_RG_THREADS) xsm[i] = p.x[i];
        for (int i = p.width + tid; i < p.K; i += LB_RG_THREADS) {
            xsm[i] = 0.f;
            if (n_vec > 1) xsm[p.K + i] = 0.f;
        }
        const bool here = mbar_wait(xbar, 0);
        if (!here && p.status) atomicExch(p.status, LB_DEV_TIMEOUT_FULL);
        __syncthreads();
        float mean = 0.f, ss = 0.f;
        if (layer_norm) {
            for (int i = tid; i < p.width; i += LB_RG_THREADS) mean += xsm[i];
            mean = block_sum(mean, red) / (float)p.width;
            for (int i = tid; i < p.width; i += LB_RG_THREADS) {
                const float d = xsm[i] - mean;
                ss += d * d;
            }
        } else {
            for (int i = tid; i < p.K / 4; i += LB_RG_THREADS) {
                const float4 v = *reinterpret_cast<const float4*>(xsm + 4 * i);
                ss += (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w);
            }
        }
        ss = block_sum(ss, red);
        const float rinv = 1.0f / sqrtf(ss / (float)p.width + p.eps), one = NORM == LB_NORM_RMS_1P ? 1.0f : 0.0f;
        if (quads) {
            auto quad = [](uint2 w) {
                return make_float4(__uint_as_float(w.x << 16), __uint_as_float(w.x & 0xffff0000u), __uint_as_float(w.y << 16), __uint_as_float(w.y & 0xffff0000u));
            };
            auto apply = [&](int i, uint2 a, uint2 b) { // quad at i with the norm weights of the one or two vectors (layer norm of one: weight, bias)
                float4 v = *reinterpret_cast<const float4*>(xsm + i);
                v.x = (v.x - mean) * rinv; v.y = (v.y - mean) * rinv; v.z = (v.z - mean) * rinv; v.w = (v.w - mean) * rinv;
                auto scaled = [&](uint2 w) {
                    const float4 f = quad(w);
                    return make_float4(v.x * (one + f.x), v.y * (one + f.y), v.z * (one + f.z), v.w * (one + f.w));
                };
                auto shift = [&](float4 r, float4 o) { return make_float4(r.x + o.x, r.y + o.y, r.z + o.z, r.w + o.w); };
                float4 r = scaled(a);
                if (layer_norm) r = shift(r, quad(n_vec > 1 ? *reinterpret_cast<const uint2*>(p.mat[0].norm_b + i) : b));
                *reinterpret_cast<float4*>(xsm + i) = r;
                if (n_vec > 1) {
                    r = scaled(b);
                    if (layer_norm) r = shift(r, quad(*reinterpret_cast<const uint2*>(p.mat[1].norm_b + i)));
                    *reinterpret_cast<float4*>(xsm + p.K + i) = r;
                }
            };
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                const int i = 4 * (tid + u * LB_RG_THREADS);
                if (i < p.width) apply(i, w_pre[0][u], w_pre[1][u]);
            }
            for (int i = 4 * (tid + 8 * LB_RG_THREADS); i < p.width; i += 4 * LB_RG_THREADS)
                apply(i, *reinterpret_cast<const uint2*>(p.mat[0].norm_w + i), second ? *reinterpret_cast<const uint2*>(second + i) : make_uint2(0u, 0u));
        } else {
            for (int i = tid; i < p.width; i += LB_RG_THREADS) {
                const float v = (xsm[i] - mean) * rinv;
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    if (e >= n_vec) continue;
                    float r = v * (one + bf16_bits_to_f32(p.mat[e].norm_w[i]));
                    if (layer_norm) r += bf16_bits_to_f32(p.mat[e].norm_b[i]);
                    xsm[e * p.K + i] = r;
                }
            }
        }
    } else {
        const int n_mix = rank == 0 ? p.n_mix : 0; // the whole mixer part lies in the first half
        const int a_lo = max(0, k_lo - p.n_mix_pad), a_hi = min(p.n_act, max(0, k_hi - p.n_mix_pad)), n_act = max(0, a_hi - a_lo);
        float* xa = xsm + (p.n_mix_pad + a_lo - k_lo);
        const int m4 = n_mix & ~3, a4 = n_act & ~3, g4 = p.gate && (reinterpret_cast<size_t>(p.gate) & 15) == 0 ? m4 : 0;
        if (tid == 0) {
            mbar_arrive_expect_tx(xbar, (uint32_t)(m4 + a4 + g4) * 4u);
            if (m4) bulk_g2s_plain(xsm, p.mix, (uint32_t)m4 * 4u, xbar);
            if (g4) bulk_g2s_plain(gate_s, p.gate, (uint32_t)g4 * 4u, xbar);
            if (a4) bulk_g2s_plain(xa, p.act + a_lo, (uint32_t)a4 * 4u, xbar);
        }
        for (int i = m4 + tid; i < n_mix; i += LB_RG_THREADS) xsm[i] = p.mix[i];
        if (p.gate)
            for (int i = g4 + tid; i < n_mix; i += LB_RG_THREADS) gate_s[i] = p.gate[i];
        for (int i = a4 + tid; i < n_act; i += LB_RG_THREADS) xa[i] = p.act[a_lo + i];
        for (int i = max(p.n_mix_pad + p.n_act, k_lo) + tid; i < k_hi; i += LB_RG_THREADS) xsm[i - k_lo] = 0.f;
        for (int i = n_mix + tid; rank == 0 && i < p.n_mix_pad; i += LB_RG_THREADS) xsm[i] = 0.f;
        const bool here = mbar_wait(xbar, 0);
        if (!here && p.status) atomicExch(p.status, LB_DEV_TIMEOUT_FULL);
        __syncthreads();
        if (p.head_w && p.gate_first) { // gate, then the norm of every part; a part is a warp's work, or everybody's when there are few
            if (p.gate)
                for (int i = tid; i < n_mix; i += LB_RG_THREADS) {
                    const float g = gate_s[i];
                    xsm[i] *= g * rg_sigmoid(g);
                }
            __syncthreads();
            const int n_part = n_mix / p.vdim, all = n_part < LB_RG_WARPS, step = all ? LB_RG_THREADS : 32, first = all ? tid : lane;
            for (int h = all ? 0 : warp; h < n_part; h += all ? 1 : LB_RG_WARPS) {
                float* o = xsm + (size_t)h * p.vdim;
                float ss = 0.f;
                for (int i = first; i < p.vdim; i += step) ss += o[i] * o[i];
                ss = all ? block_sum(ss, red) : warp_sum(ss);
                const float rinv = 1.0f / sqrtf(ss / (float)p.vdim + p.eps);
                for (int i = first; i < p.vdim; i += step) o[i] *= rinv * bf16_bits_to_f32(__ldg(p.head_w + (size_t)h * p.vdim + i));
            }
        } else if (p.head_w) {
            const int heads = n_mix / p.vdim;
            for (int h = warp; h < heads; h += LB_RG_WARPS) {
                float* o = xsm + (size_t)h * p.vdim;
                float ss = 0.f;
                for (int i = lane; i < p.vdim; i += 32) ss += o[i] * o[i];
                const float rinv = 1.0f / sqrtf(warp_sum(ss) / (float)p.vdim + p.eps);
                for (int i = lane; i < p.vdim; i += 32) {
                    float v = o[i] * rinv * bf16_bits_to_f32(__ldg(p.head_w + i));
                    if (p.gate) {
                        const float g = gate_s[h * p.vdim + i];
                        v *= g * rg_sigmoid(g);
                    }
                    o[i] = v;
                }
            }
        }
    }
    __syncthreads();
    pdl_launch_dependents();

    int slot = 0;
    uint32_t phase = 0;
    bool ok = true;
    for (int item = warp; item < items && ok; item += LB_RG_WARPS) {
        const int pair = split == 1 ? item : item / split, seg0 = seg_lo + (item - pair * split) * spp;
        const float* xv = xsm + ((n_vec > 1 && c + pair * G >= pairs0) ? p.K : 0) - k_lo;
        float a0 = 0.f, a1 = 0.f, b0 = 0.f, b1 = 0.f;
        for (int s = 0; s < spp; ++s) {
            if (!__all_sync(0xffffffffu, mbar_wait(&bars[warp * S + slot], phase))) { // bounded: the rows left keep their old result
                if (lane == 0 && p.status) atomicExch(p.status, LB_DEV_TIMEOUT_FULL);
                ok = false;
                break;
            }
            int k0, len, e;
            segment(seg0 + s, k0, len, e);
            const int n8 = len >> 3;
            const uint4* wa = reinterpret_cast<const uint4*>(ring + (size_t)(warp * S + slot) * (LB_RG_SEG * 4));
            const uint4* wb = wa + LB_RG_SEG / 8;
#pragma unroll 4
            for (int i = lane; i < n8; i += 32) {
                const uint4 u = wa[i], v = wb[i];
                const float4 x0 = *reinterpret_cast<const float4*>(xv + k0 + i * 8), x1 = *reinterpret_cast<const float4*>(xv + k0 + i * 8 + 4);
                a0 = fmaf(__uint_as_float(u.x << 16), x0.x, a0);
                a1 = fmaf(__uint_as_float(u.x & 0xffff0000u), x0.y, a1);
                b0 = fmaf(__uint_as_float(v.x << 16), x0.x, b0);
                b1 = fmaf(__uint_as_float(v.x & 0xffff0000u), x0.y, b1);
                a0 = fmaf(__uint_as_float(u.y << 16), x0.z, a0);
                a1 = fmaf(__uint_as_float(u.y & 0xffff0000u), x0.w, a1);
                b0 = fmaf(__uint_as_float(v.y << 16), x0.z, b0);
                b1 = fmaf(__uint_as_float(v.y & 0xffff0000u), x0.w, b1);
                a0 = fmaf(__uint_as_float(u.z << 16), x1.x, a0);
                a1 = fmaf(__uint_as_float(u.z & 0xffff0000u), x1.y, a1);
                b0 = fmaf(__uint_as_float(v.z << 16), x1.x, b0);
                b1 = fmaf(__uint_as_float(v.z & 0xffff0000u), x1.y, b1);
                a0 = fmaf(__uint_as_float(u.w << 16), x1.z, a0);
                a1 = fmaf(__uint_as_float(u.w & 0xffff0000u), x1.w, a1);
                b0 = fmaf(__uint_as_float(v.w << 16), x1.z, b0);
                b1 = fmaf(__uint_as_float(v.w & 0xffff0000u), x1.w, b1);
            }
            __syncwarp(); // every lane has its words in registers (the sums depend on them): the slot can be refilled
            request();    // the slot just freed is the next one the request cursor fills
            if (++slot == S) { slot = 0; phase ^= 1u; }
        }
        const float ya = warp_sum(a0 + a1), yb = warp_sum(b0 + b1);
        if (lane == 0) { part[2 * item] = ya; part[2 * item + 1] = yb; }
    }
    bool all_ok = __syncthreads_and(ok ? 1 : 0) != 0;
    if (KS > 1) { // this half's sums where the other CTA finds them
        for (int m = tid; m < my_pairs; m += LB_RG_THREADS) {
            float2 r = make_float2(0.f, 0.f);
            for (int q = 0; q < split; ++q) {
                r.x += part[2 * (m * split + q)];
                r.y += part[2 * (m * split + q) + 1];
            }
            *reinterpret_cast<float2*>(part + 2 * m * split) = r; // read and written by this thread alone
        }
        if (tid == 0) red[36] = all_ok ? 1.f : 0.f;
        if (tid == 0) red[37] = (float)split;
        rg_cluster_sync();
        all_ok = rg_ld_cluster(red + 36, rank ^ 1).x != 0.f && all_ok;
    }
    const int other_split = KS > 1 ? (int)rg_ld_cluster(red + 36, rank ^ 1).y : 0;

    float best_v = -INFINITY;
    int best_i = 0x7fffffff;
    for (int m = tid; m < my_pairs && all_ok; m += LB_RG_THREADS) {
        float r[2] = {0.f, 0.f};
        if (KS > 1) {
            if ((m & 1) != rank) continue; // the two CTAs finish every other pair each
            const float2 mine = *reinterpret_cast<const float2*>(part + 2 * m * split), his = rg_ld_cluster(part + 2 * m * other_split, rank ^ 1);
            r[0] = rank == 0 ? mine.x + his.x : his.x + mine.x;
            r[1] = rank == 0 ? mine.y + his.y : his.y + mine.y;
        } else {
            for (int q = 0; q < split; ++q) {
                r[0] += part[2 * (m * split + q)];
                r[1] += part[2 * (m * split + q) + 1];
            }
        }
        const int g = c + m * G, mi = g >= pairs0, n = 2 * (mi ? g - pairs0 : g);
        const lb_rg_mat& M = p.mat[mi];
        if (M.y_mode == LB_DY_RELU_GLU) {
            M.y[n >> 1] = fmaxf(r[0], 0.f) * r[1];
        } else if (M.y_mode == LB_DY_CLAMP_GLU) {
            const int part = SEL ? n / p.sel_rows : 0, i = (n - part * p.sel_rows) >> 1;
            const float ga = fminf(r[0], p.limit), up = fminf(fmaxf(r[1], -p.limit), p.limit);
            M.y[(size_t)part * p.y_part + i] = ga * rg_sigmoid(p.alpha * ga) * (up + 1.0f);
        } else {
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                if (n + e >= M.rows) continue;
                float v = r[e];
                if (M.y_mode == LB_DY_RESIDUAL) v = fmaf(p.mult, v, M.y[n + e]);
                else if (M.y_mode == LB_DY_SOFTCAP && p.cap > 0.f) v = p.cap * tanhf(v / p.cap);
                else if (M.y_mode == LB_DY_RELU2) v = fmaxf(v, 0.f) * fmaxf(v, 0.f);
                M.y[n + e] = v;
                if (v > best_v || (v == best_v && n + e < best_i)) { best_v = v; best_i = n + e; }
            }
        }
    }
    if (p.part_val) { // this CTA's candidate for the arg-max: greater value, smaller row on ties
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, best_v, o);
            const int oi = __shfl_xor_sync(0xffffffffu, best_i, o);
            if (ov > best_v || (ov == best_v && oi < best_i)) { best_v = ov; best_i = oi; }
        }
        int* ri = reinterpret_cast<int*>(red + 16);
        if (lane == 0) { red[warp] = best_v; ri[warp] = best_i; }
        __syncthreads();
        if (tid == 0) {
            for (int w = 1; w < LB_RG_WARPS; ++w)
                if (red[w] > best_v || (red[w] == best_v && ri[w] < best_i)) { best_v = red[w]; best_i = ri[w]; }
            p.part_val[c] = best_v;
            p.part_idx[c] = best_i;
        }
    }
    if (KS > 1) rg_cluster_sync(); // nobody leaves while the other CTA still reads its sums
}
#define RG_KERNEL(name, NORM, SEL)                                                                                                     \
    extern "C" __global__ void __launch_bounds__(LB_RG_THREADS, 1) name(const __grid_constant__ lb_rows_gemv_params p) { \
        rows_gemv_body<NORM, SEL>(p);                                                                                                  \
    }
RG_KERNEL(rows_gemv, LB_NORM_RMS_1P, false)
RG_KERNEL(rows_gemv_rms, LB_NORM_RMS, false)
RG_KERNEL(rows_gemv_ln, LB_NORM_LAYER, false)
RG_KERNEL(rows_gemv_experts, LB_NORM_LAYER, true)
