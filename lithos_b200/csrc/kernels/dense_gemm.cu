// Dense products of a prompt chunk for bf16 models: Y[T, N] = X[T, K] W[N, K]^T with fused epilogues, one or two of them (the mixer's
// and the feed-forward's input projections read differently normed copies of the same rows) in one launch; and the chunk's RMS norm.
//
// gemm_bf16_tc: 5th-generation tensor cores.  A tile is 128 weight rows x NT (16..256) tokens: tcgen05.mma 128 x NT x 16, both operands by
// tiled TMA (64 k x rows, 128-byte swizzle), accumulators in tensor memory.  Persistent CTAs of six warps: one lane brings operands, one
// lane issues products, four warps read accumulators (lane = weight row, column = token) and finish them.  Two accumulators, so the
// epilogue of a tile runs beside the products of the next.  Weight rows are the lanes, so 32 neighbouring outputs of a token are one
// coalesced store and a (gate, up) pair sits in neighbouring lanes.  Every wait is bounded and reports through the status word.
// With experts the chunk's (token, expert) assignments come sorted by expert (moe_plan) and every token tile belongs to one of them.
// gemm_f32_simt: the same products in fp32 throughout (fp32 activations, weights exact in fp32, fp32 fused multiply-adds).
#include "tcgen05.cuh"
#include "params.h"

#define DG_FAIL_EMPTY 0x1201u // status: a stage's products never completed
#define DG_FAIL_FULL 0x1202u  // status: a stage's operands never landed
#define DG_FAIL_ACC 0x1203u   // status: an accumulator was never completed / never freed

__device__ __forceinline__ void dg_tma(uint32_t dst_smem, const void* tmap, int k, int row, uint64_t* bar) {
    asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(dst_smem),
                 "l"(tmap), "r"(k), "r"(row), "r"(smem_u32(bar))
                 : "memory");
}

// tile t of a launch: product m, weight rows from row (row in its matrix: n0), tokens tok .. end - 1.  With experts a token tile is an entry
// of the plan and the expert's rows are rows of the stack.
struct dg_tile { int m, row, n0, tok, end; };
__device__ __forceinline__ dg_tile dg_find(const lb_dgemm_params& p, int t) {
    dg_tile d;
    if (p.plan_tiles) {
        const int tt = t / p.tiles[0];
        const int4 e = __ldg(reinterpret_cast<const int4*>(p.plan_tiles) + tt);
        d.m = 0;
        d.n0 = (t - tt * p.tiles[0]) * LB_DG_ROWS;
        d.row = e.x * p.expert_rows + d.n0;
        d.tok = e.y;
        d.end = e.z;
    } else {
        const int rt = t / p.t_tiles, tt = t - rt * p.t_tiles;
        d.m = rt >= p.tiles[0];
        d.row = d.n0 = (d.m ? rt - p.tiles[0] : rt) * LB_DG_ROWS;
        d.tok = tt * p.NT;
        d.end = p.T;
    }
    return d;
}
__device__ __forceinline__ float dg_clamp_glu(float gate, float up, float limit, float alpha) {
    const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
    return g / (1.0f + expf(-alpha * g)) * (u + 1.0f);
}

// a warp's 32 weight rows (lane: row n) x n_t tokens from t0 on: out of tensor memory, finished, stored
template <int MODE>
__device__ __forceinline__ void dg_finish(const lb_dgemm_params& p, int m, uint32_t acc, int n, int t0, int n_t, int ld) {
    const int lane = threadIdx.x & 31;
    const bool live = n < p.rows[m];
    const int hn = MODE == LB_DY_HEADS ? n / p.head[m] : 0, col = MODE == LB_DY_HEADS ? hn * p.head_p[m] + (n - hn * p.head[m]) : n;
    for (int c = 0; c < n_t; c += 16) {
        uint32_t r[16];
        tmem_ld16(acc + (uint32_t)c, r);
        tmem_ld_wait();
        if (MODE == LB_DY_HEADS || MODE == LB_DY_RELU2) {
#pragma unroll
            for (int j = 0; j < 16; ++j) {
                if (!live || c + j >= n_t) continue;
                float v = __uint_as_float(r[j]);
                if (MODE == LB_DY_RELU2) v = fmaxf(v, 0.f) * fmaxf(v, 0.f);
                const size_t o = (size_t)(t0 + c + j) * ld + col;
                if (MODE == LB_DY_RELU2 && p.y_f32[m]) reinterpret_cast<float*>(p.y[m])[o] = v;
                else reinterpret_cast<__nv_bfloat16*>(p.y[m])[o] = __float2bfloat16_rn(v);
            }
        } else if (MODE == LB_DY_RELU_GLU || MODE == LB_DY_CLAMP_GLU) {
            const bool st = live && !(lane & 1);
#pragma unroll
            for (int j = 0; j < 16; ++j) {
                const float gate = __uint_as_float(r[j]), up = __uint_as_float(__shfl_xor_sync(0xffffffffu, r[j], 1));
                const float v = MODE == LB_DY_RELU_GLU ? fmaxf(gate, 0.f) * up : dg_clamp_glu(gate, up, p.limit, p.alpha);
                if (st && c + j < n_t) {
                    const size_t o = (size_t)(t0 + c + j) * ld + (n >> 1);
                    if (p.y_f32[m]) reinterpret_cast<float*>(p.y[m])[o] = v;
                    else reinterpret_cast<__nv_bfloat16*>(p.y[m])[o] = __float2bfloat16_rn(v);
                }
            }
        } else {
            float* y = reinterpret_cast<float*>(p.y[m]) + (size_t)(t0 + c) * ld + n;
            float old[16];
            if (MODE == LB_DY_RESIDUAL) {
#pragma unroll
                for (int j = 0; j < 16; ++j) old[j] = live && c + j < n_t ? y[(size_t)j * ld] : 0.f;
            }
#pragma unroll
            for (int j = 0; j < 16; ++j) {
                float v = __uint_as_float(r[j]);
                if (MODE == LB_DY_RESIDUAL) v = fmaf(p.mult, v, old[j]);
                else if (MODE == LB_DY_SOFTCAP && p.cap > 0.f) v = p.cap * tanhf(v / p.cap);
                if (live && c + j < n_t) y[(size_t)j * ld] = v;
            }
        }
    }
}

extern "C" __global__ void __launch_bounds__(LB_DG_THREADS, 1) gemm_bf16_tc(const __grid_constant__ lb_dgemm_params p) {
    extern __shared__ __align__(1024) unsigned char dg_sm[];
    __shared__ __align__(8) uint64_t bar_full[LB_DG_MAX_STAGES], bar_empty[LB_DG_MAX_STAGES], bar_acc[2], bar_free[2];
    __shared__ uint32_t tmem_slot;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int S = p.stages, NT = p.NT;
    const uint32_t a_bytes = LB_DG_ROWS * LB_DG_KB * 2, b_bytes = (uint32_t)NT * LB_DG_KB * 2, stage_bytes = a_bytes + b_bytes;
    const int ksteps = p.K / LB_DG_KB;
    if (tid == 0) {
        for (int s = 0; s < S; ++s) {
            mbar_init(&bar_full[s], 1);
            mbar_init(&bar_empty[s], 1);
        }
        for (int s = 0; s < 2; ++s) {
            mbar_init(&bar_acc[s], 1);
            mbar_init(&bar_free[s], 4);
        }
        mbar_fence_init();
    }
    if (warp == 1) tmem_alloc(&tmem_slot, (uint32_t)p.tmem_cols);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_slot;
    pdl_wait();
    const int n_tiles = p.plan_tiles ? p.plan_n[0] * p.tiles[0] : (p.tiles[0] + p.tiles[1]) * p.t_tiles;

    if (warp == 0 && lane == 0) {
        // ---------------- operands ----------------
        int s = 0, issued = 0;
        uint32_t ph = 0;
        bool ok = true;
        for (int tile = blockIdx.x; tile < n_tiles && ok; tile += gridDim.x) {
            const dg_tile d = dg_find(p, tile);
            for (int k = 0; k < ksteps; ++k) {
                if (issued >= S && !tc_wait(&bar_empty[s], ph ^ 1u)) {
                    ok = false;
                    if (p.status) atomicExch(p.status, DG_FAIL_EMPTY);
                    break;
                }
                mbar_arrive_expect_tx(&bar_full[s], stage_bytes);
                const uint32_t dst = smem_u32(dg_sm) + (uint32_t)s * stage_bytes;
                dg_tma(dst, p.tmap_w[d.m], k * LB_DG_KB, d.row, &bar_full[s]);
                dg_tma(dst + a_bytes, p.tmap_x[d.m], k * LB_DG_KB, d.tok, &bar_full[s]);
                ++issued;
                if (++s == S) { s = 0; ph ^= 1u; }
            }
        }
        if (!ok) // nothing may still be on its way into this CTA's shared memory when it ends
            for (int i = 0; i < S && i < issued; ++i) {
                if (--s < 0) { s = S - 1; ph ^= 1u; }
                tc_wait(&bar_full[s], ph);
            }
    } else if (warp == 1 && lane == 0) {
        // ---------------- products ----------------
        const uint32_t idesc = tc_idesc_bf16(LB_DG_ROWS, (uint32_t)NT);
        int s = 0, it = 0;
        uint32_t ph = 0;
        bool ok = true;
        for (int tile = blockIdx.x; tile < n_tiles && ok; tile += gridDim.x, ++it) {
            const int b = it & 1;
            if (it >= 2 && !tc_wait(&bar_free[b], (uint32_t)((it >> 1) - 1) & 1u)) { // the epilogue has read this accumulator
                ok = false;
                if (p.status) atomicExch(p.status, DG_FAIL_ACC);
                break;
            }
            tc_fence_after();
            const uint32_t d = tmem + (uint32_t)(b * NT);
            for (int k = 0; k < ksteps; ++k) {
                if (!tc_wait(&bar_full[s], ph)) {
                    ok = false;
                    if (p.status) atomicExch(p.status, DG_FAIL_FULL);
                    break;
                }
                tc_fence_after();
                const uint32_t base = smem_u32(dg_sm) + (uint32_t)s * stage_bytes;
                const uint64_t ad = tc_smem_desc(base, 16, 1024), bd = tc_smem_desc(base + a_bytes, 16, 1024);
#pragma unroll
                for (int kk = 0; kk < LB_DG_KB / 16; ++kk)
                    tc_mma(d, ad + (uint64_t)(kk * 2), bd + (uint64_t)(kk * 2), idesc, (k > 0 || kk > 0) ? 1u : 0u);
                tc_commit(&bar_empty[s]);
                if (++s == S) { s = 0; ph ^= 1u; }
            }
            if (ok) tc_commit(&bar_acc[b]);
        }
    } else if (warp >= 2) {
        // ---------------- epilogue: warp w reads the tensor-memory lanes 32 (w % 4) .. + 31 ----------------
        const int quad = warp & 3;
        int it = 0;
        for (int tile = blockIdx.x; tile < n_tiles; tile += gridDim.x, ++it) {
            const int b = it & 1;
            const dg_tile d = dg_find(p, tile);
            const int m = d.m, n = d.n0 + quad * 32 + lane, t0 = d.tok;
            const bool got = tc_wait(&bar_acc[b], (uint32_t)(it >> 1) & 1u);
            if (!__all_sync(0xffffffffu, got)) {
                if (lane == 0 && p.status) atomicExch(p.status, DG_FAIL_ACC);
                break;
            }
            tc_fence_after();
            const int mode = p.y_mode[m], ld = p.ld_y[m], n_t = min(NT, d.end - t0);
            const uint32_t acc = tmem + ((uint32_t)(32 * quad) << 16) + (uint32_t)(b * NT);
            switch (mode) {
                case LB_DY_RELU_GLU: dg_finish<LB_DY_RELU_GLU>(p, m, acc, n, t0, n_t, ld); break;
                case LB_DY_CLAMP_GLU: dg_finish<LB_DY_CLAMP_GLU>(p, m, acc, n, t0, n_t, ld); break;
                case LB_DY_RELU2: dg_finish<LB_DY_RELU2>(p, m, acc, n, t0, n_t, ld); break;
                case LB_DY_HEADS: dg_finish<LB_DY_HEADS>(p, m, acc, n, t0, n_t, ld); break;
                case LB_DY_RESIDUAL: dg_finish<LB_DY_RESIDUAL>(p, m, acc, n, t0, n_t, ld); break;
                case LB_DY_SOFTCAP: dg_finish<LB_DY_SOFTCAP>(p, m, acc, n, t0, n_t, ld); break;
                default: dg_finish<LB_DY_STORE>(p, m, acc, n, t0, n_t, ld); break;
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&bar_free[b]);
        }
    }
    pdl_launch_dependents();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc(tmem, (uint32_t)p.tmem_cols);
    }
}

// ---- fp32 ----------------------------------------------------------------------------------------------------------
#define SG_TN 64 // weight rows per tile
#define SG_TT 64 // tokens per tile
#define SG_KB 16
// grid (row tiles of both products, token tiles), block 256: a thread owns 4 rows x 4 tokens.  K is a multiple of 64.
extern "C" __global__ void __launch_bounds__(256) gemm_f32_simt(const __grid_constant__ lb_dgemm_params p) {
    __shared__ __align__(16) float ws[SG_KB][SG_TN + 4], xs[SG_KB][SG_TT + 4];
    pdl_wait();
    const int tid = threadIdx.x, tn = tid & 15, tt = tid >> 4;
    const int nt0 = (p.rows[0] + SG_TN - 1) / SG_TN, m = (int)blockIdx.x >= nt0;
    const int row0 = ((int)blockIdx.x - (m ? nt0 : 0)) * SG_TN;
    int t0 = blockIdx.y * SG_TT, end = p.T;
    const uint16_t* W = p.w[m];
    if (p.plan_tiles) {
        if ((int)blockIdx.y >= p.plan_n[0]) return;
        const int4 e = reinterpret_cast<const int4*>(p.plan_tiles)[blockIdx.y];
        W += (size_t)e.x * p.expert_rows * p.K;
        t0 = e.y;
        end = e.z;
    }
    const float* X = reinterpret_cast<const float*>(p.x[m]);
    float acc[4][4] = {};
    const int lr = tid >> 2, lk = (tid & 3) * 4; // load: row / token of the tile, 4 k
    for (int k0 = 0; k0 < p.K; k0 += SG_KB) {
        uint2 w = make_uint2(0u, 0u);
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
        if (row0 + lr < p.rows[m]) w = *reinterpret_cast<const uint2*>(W + (size_t)(row0 + lr) * p.K + k0 + lk);
        if (t0 + lr < end) x = *reinterpret_cast<const float4*>(X + (size_t)(t0 + lr) * p.ld_x + k0 + lk);
        __syncthreads();
        ws[lk][lr] = __uint_as_float(w.x << 16);
        ws[lk + 1][lr] = __uint_as_float(w.x & 0xffff0000u);
        ws[lk + 2][lr] = __uint_as_float(w.y << 16);
        ws[lk + 3][lr] = __uint_as_float(w.y & 0xffff0000u);
        xs[lk][lr] = x.x;
        xs[lk + 1][lr] = x.y;
        xs[lk + 2][lr] = x.z;
        xs[lk + 3][lr] = x.w;
        __syncthreads();
#pragma unroll
        for (int k = 0; k < SG_KB; ++k) {
            const float4 a = *reinterpret_cast<const float4*>(&ws[k][tn * 4]), b = *reinterpret_cast<const float4*>(&xs[k][tt * 4]);
            const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
        }
    }
    pdl_launch_dependents();
    const int mode = p.y_mode[m], ld = p.ld_y[m];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const int t = t0 + tt * 4 + j;
        if (t >= end) continue;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int n = row0 + tn * 4 + i;
            if (n >= p.rows[m]) continue;
            float v = acc[i][j];
            float* y = reinterpret_cast<float*>(p.y[m]) + (size_t)t * ld;
            if (mode == LB_DY_RELU_GLU) {
                if (i & 1) continue;
                v = fmaxf(v, 0.f) * acc[i | 1][j];
                if (p.y_f32[m]) y[n >> 1] = v;
                else reinterpret_cast<__nv_bfloat16*>(p.y[m])[(size_t)t * ld + (n >> 1)] = __float2bfloat16_rn(v);
            } else if (mode == LB_DY_CLAMP_GLU) {
                if (!(i & 1)) y[n >> 1] = dg_clamp_glu(v, acc[i | 1][j], p.limit, p.alpha);
            } else if (mode == LB_DY_RELU2) y[n] = fmaxf(v, 0.f) * fmaxf(v, 0.f);
            else if (mode == LB_DY_RESIDUAL) y[n] = fmaf(p.mult, v, y[n]);
            else y[n] = mode == LB_DY_SOFTCAP && p.cap > 0.f ? p.cap * tanhf(v / p.cap) : v;
        }
    }
}

// norm of a chunk's rows (lb_norm2_params), columns width..ld are zero.  grid T, block 256.  Rows of whole quads up to
// 4 NR_Q x 256 columns stay in registers between the passes.
#define NR_Q 8
__device__ __forceinline__ float4 nr_quad(const uint16_t* w, int i) {
    const uint2 u = __ldg(reinterpret_cast<const uint2*>(w + i));
    return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16), __uint_as_float(u.y & 0xffff0000u));
}
__device__ __forceinline__ float nr_added(const lb_norm2_params& p, int t, int i) { // sum of the token's rows of y, in the order of its parts
    float s = 0.f;
    for (int k = 0; k < p.y_top; ++k) {
        const size_t o = (size_t)p.y_place[(size_t)t * p.y_top + k] * p.ld_y + i;
        s += p.f32 ? reinterpret_cast<const float*>(p.y)[o] : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p.y)[o]);
    }
    return s;
}
__device__ __forceinline__ void nr_store4(const lb_norm2_params& p, void* h, size_t o, float4 r) {
    if (p.f32) *reinterpret_cast<float4*>(reinterpret_cast<float*>(h) + o) = r;
    else {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(r.x, r.y), hi = __floats2bfloat162_rn(r.z, r.w);
        *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(h) + o) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
    }
}
__device__ __forceinline__ void nr_store1(const lb_norm2_params& p, void* h, size_t o, float r) {
    if (p.f32) reinterpret_cast<float*>(h)[o] = r;
    else reinterpret_cast<__nv_bfloat16*>(h)[o] = __float2bfloat16_rn(r);
}
// ANY false: LB_NORM_RMS_1P of rows of `width`, nothing added, nothing scattered
template <bool ANY>
__device__ __forceinline__ void norm_rows2_body(const lb_norm2_params& p) {
    __shared__ float red[40];
    const int t = threadIdx.x, tok = blockIdx.x;
    const bool quads = (p.width & 3) == 0 && (!ANY || ((p.ld_x & 3) == 0 && (p.ld_y & 3) == 0)) && p.width <= 4 * NR_Q * 256;
    const float one = !ANY || p.norm == LB_NORM_RMS_1P ? 1.0f : 0.0f;
    const bool layer_norm = ANY && p.norm == LB_NORM_LAYER, adds = ANY && p.y, scatters = ANY && p.scatter;
    pdl_wait();
    float* x = p.x + (size_t)tok * (ANY ? p.ld_x : p.width);
    float4 v[NR_Q];
    float mean = 0.f, ss = 0.f;
    if (quads) {
#pragma unroll
        for (int u = 0; u < NR_Q; ++u) {
            const int i = 4 * (t + 256 * u);
            v[u] = i < p.width ? *reinterpret_cast<const float4*>(x + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
        if (adds) {
#pragma unroll
            for (int u = 0; u < NR_Q; ++u) {
                const int i = 4 * (t + 256 * u);
                if (i >= p.width) continue;
                float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
                for (int k = 0; k < p.y_top; ++k) {
                    const size_t o = (size_t)p.y_place[(size_t)tok * p.y_top + k] * p.ld_y + i;
                    const float4 a = p.f32 ? *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p.y) + o) : nr_quad(reinterpret_cast<const uint16_t*>(p.y) + o, 0);
                    s.x += a.x; s.y += a.y; s.z += a.z; s.w += a.w;
                }
                v[u].x = fmaf(p.y_mult, s.x, v[u].x); v[u].y = fmaf(p.y_mult, s.y, v[u].y);
                v[u].z = fmaf(p.y_mult, s.z, v[u].z); v[u].w = fmaf(p.y_mult, s.w, v[u].w);
                *reinterpret_cast<float4*>(x + i) = v[u];
            }
        }
        if (layer_norm) {
#pragma unroll
            for (int u = 0; u < NR_Q; ++u) mean += (v[u].x + v[u].y) + (v[u].z + v[u].w);
            mean = block_sum(mean, red) / (float)p.width;
#pragma unroll
            for (int u = 0; u < NR_Q; ++u)
                if (4 * (t + 256 * u) < p.width) { v[u].x -= mean; v[u].y -= mean; v[u].z -= mean; v[u].w -= mean; }
        }
#pragma unroll
        for (int u = 0; u < NR_Q; ++u) ss += (v[u].x * v[u].x + v[u].y * v[u].y) + (v[u].z * v[u].z + v[u].w * v[u].w);
    } else {
        if (adds)
            for (int i = t; i < p.width; i += 256) x[i] = fmaf(p.y_mult, nr_added(p, tok, i), x[i]); // read again by this thread alone
        if (layer_norm) {
            for (int i = t; i < p.width; i += 256) mean += x[i];
            mean = block_sum(mean, red) / (float)p.width;
        }
#pragma unroll 4
        for (int i = t; i < p.width; i += 256) {
            const float d = x[i] - mean;
            ss += d * d;
        }
    }
    ss = block_sum(ss, red);
    const float rinv = 1.0f / sqrtf(ss / (float)p.width + p.eps);
    pdl_launch_dependents();
    if (ANY && !p.h[0]) return; // only the sum was asked for
    const int copies = scatters ? p.top : 1;
    if (quads) {
#pragma unroll
        for (int u = 0; u < NR_Q; ++u) {
            const int i = 4 * (t + 256 * u);
            if (i >= p.width) continue;
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                if (!p.h[e]) continue;
                const float4 w = nr_quad(p.w[e], i);
                float4 r = make_float4(v[u].x * rinv * (one + w.x), v[u].y * rinv * (one + w.y), v[u].z * rinv * (one + w.z), v[u].w * rinv * (one + w.w));
                if (layer_norm) {
                    const float4 b = nr_quad(p.b[e], i);
                    r.x += b.x; r.y += b.y; r.z += b.z; r.w += b.w;
                }
                for (int k = 0; k < copies; ++k) nr_store4(p, p.h[e], (size_t)(scatters ? p.scatter[(size_t)tok * p.top + k] : tok) * p.ld + i, r);
            }
        }
    }
    for (int i = quads ? p.width + t : t; i < p.ld; i += 256) {
        const float xv = i < p.width ? (x[i] - mean) * rinv : 0.f;
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            if (!p.h[e]) continue;
            float r = i < p.width ? xv * (one + bf16_bits_to_f32(p.w[e][i])) : 0.f;
            if (layer_norm && i < p.width) r += bf16_bits_to_f32(p.b[e][i]);
            for (int k = 0; k < copies; ++k) nr_store1(p, p.h[e], (size_t)(scatters ? p.scatter[(size_t)tok * p.top + k] : tok) * p.ld + i, r);
        }
    }
}
extern "C" __global__ void __launch_bounds__(256, 4) norm_rows2(const __grid_constant__ lb_norm2_params p) { norm_rows2_body<false>(p); }
extern "C" __global__ void __launch_bounds__(256, 4) norm_rows_any(const __grid_constant__ lb_norm2_params p) { norm_rows2_body<true>(p); }

// The chunk's (token, expert) assignments sorted by expert: the row of every assignment, and the token tiles (of at most NT assignments of one
// expert).  One CTA of 1024 threads per launch.
extern "C" __global__ void __launch_bounds__(1024) moe_plan(const __grid_constant__ lb_moe_plan_params p) {
    __shared__ int count[LB_MOE_MAX_EXPERTS], first[LB_MOE_MAX_EXPERTS], tile0[LB_MOE_MAX_EXPERTS], wsum[2][32];
    const int t = threadIdx.x, n = p.T * p.top, lane = t & 31, warp = t >> 5;
    count[t] = 0;
    __syncthreads();
    pdl_wait(); // the buffers written here may still be read by the kernels before
    auto expert = [&](int a) {
        const int s = a / p.top;
        return p.table[(size_t)p.tokens[s] * p.top + (a - s * p.top)];
    };
    for (int a0 = t; a0 < n; a0 += 8 * 1024) { // the reads of eight assignments, then their places among their experts' ones
        int e[8];
#pragma unroll
        for (int k = 0; k < 8; ++k) e[k] = a0 + k * 1024 < n ? expert(a0 + k * 1024) : -1;
#pragma unroll
        for (int k = 0; k < 8; ++k)
            if (e[k] >= 0) p.place[a0 + k * 1024] = atomicAdd(&count[e[k]], 1);
    }
    __syncthreads();
    // exclusive sums over experts of assignments and of tiles
    const int c = t < p.experts ? count[t] : 0, nt = (c + p.NT - 1) / p.NT;
    int ic = c, it = nt;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const int a = __shfl_up_sync(0xffffffffu, ic, o), b = __shfl_up_sync(0xffffffffu, it, o);
        if (lane >= o) { ic += a; it += b; }
    }
    if (lane == 31) { wsum[0][warp] = ic; wsum[1][warp] = it; }
    __syncthreads();
    int bc = 0, bt = 0;
    for (int w = 0; w < warp; ++w) { bc += wsum[0][w]; bt += wsum[1][w]; }
    first[t] = bc + ic - c;
    tile0[t] = bt + it - nt;
    if (t == 1023) p.n_tiles[0] = bt + it;
    for (int k = 0; k < nt; ++k) reinterpret_cast<int4*>(p.tiles)[tile0[t] + k] = make_int4(t, first[t] + k * p.NT, first[t] + c, 0);
    __syncthreads();
    for (int a0 = t; a0 < n; a0 += 8 * 1024) {
        int e[8], q[8];
#pragma unroll
        for (int k = 0; k < 8; ++k) {
            e[k] = a0 + k * 1024 < n ? expert(a0 + k * 1024) : -1;
            q[k] = e[k] >= 0 ? p.place[a0 + k * 1024] : 0;
        }
#pragma unroll
        for (int k = 0; k < 8; ++k)
            if (e[k] >= 0) p.place[a0 + k * 1024] = q[k] + first[e[k]];
    }
    pdl_launch_dependents();
}
