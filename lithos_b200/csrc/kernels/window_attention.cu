// Attention for layers with general head sizes (up to 256), positions seen in blocks, rotated values and a soft-max sink:
//   q, k: the first rot_dims features rotate by position in neighbouring pairs; v: divided by its root mean square, then all of it
//   rotated by its position; weight of key j at position i = exp(s_ij) / (sink + sum exp(s)), s = scale q.k, over the keys j <= i of i's
//   block of positions; the weighted sum of values is rotated back by i.
// The cache holds rotated keys and normed, rotated values, so a layer can attend over another layer's cache (k_off < 0).
// Scores, weights and sums are fp32; angles are reduced in double.
//   wattn_rows_*   one query token per CTA row: the decode step (positions cut into slices merged by the last CTA), and prompts in fp32
//   wattn_prepare  a prompt chunk's keys and values into the cache; its queries as two bf16 terms
//   wattn_chunk_*  a prompt chunk on the tensor cores
#include "mma_sync.cuh"
#include "rotate.cuh"

struct wa_angles { // cosines and sines of a position: key / query pairs and value pairs
    float ck[LB_WA_MAX_DIM / 2], sk[LB_WA_MAX_DIM / 2], cv[LB_WA_MAX_DIM / 2], sv[LB_WA_MAX_DIM / 2];
};
__device__ __forceinline__ void wa_fill_angles(const lb_wattn_params& p, int pos, wa_angles& A) {
    for (int i = threadIdx.x; i < p.rot_dims / 2; i += blockDim.x) wa_angle(p.freq_k[i], pos, A.ck[i], A.sk[i]);
    if (p.freq_v)
        for (int i = threadIdx.x; i < p.vdim / 2; i += blockDim.x) wa_angle(p.freq_v[i], pos, A.cv[i], A.sv[i]);
}
template <typename T>
__device__ __forceinline__ void wa_warp_value(const lb_wattn_params& p, const float* src, T* dst, const wa_angles& A) {
    float r = 1.f;
    if (p.v_norm) {
        float ss = 0.f;
        for (int i = threadIdx.x & 31; i < p.vdim; i += 32) ss += src[i] * src[i];
        r = 1.0f / sqrtf(warp_sum(ss) / (float)p.vdim + p.eps);
    }
    wa_warp_rotate(src, dst, p.vdim, p.freq_v ? p.vdim : 0, A.cv, A.sv, r);
}

#define WR_MAX_WARPS 4
// grid (KV * groups, splits, tokens), block 32 x warps (1..4); GH query heads per CTA, NV pairs of value features per lane (64 NV >= vdim).
// A warp takes tiles of 32 cache rows: the tile's K and V rows come to shared memory in one go, a lane scores one row for all heads of the
// CTA (no exchange between lanes), then lanes own value features.  In the decode step everything that does not depend on this step's
// projections -- position, angles, the first tile (rows of earlier positions, written by kernels that have long finished) -- is under way
// before the wait for the previous kernel.
// dynamic shared memory: q [GH][dim_p] fp32 | accumulators [warps][GH][vdim_p] fp32 | new key, value row in the cache's format |
// tiles [warps][32][K row + 16 B, V row + 16 B]
template <typename TC, int GH, int NV>
__device__ __forceinline__ void wattn_rows_body(const lb_wattn_params& p) {
    extern __shared__ __align__(16) unsigned char wr_sm[];
    __shared__ wa_angles A;
    __shared__ __align__(16) float pw[WR_MAX_WARPS][32][GH];
    __shared__ float ml[WR_MAX_WARPS][GH][2];
    __shared__ float fw[LB_WA_MAX_SPLITS][GH]; // weight of each slice (or warp) in the merged sum, denominators divided in
    __shared__ int last_flag;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nw = blockDim.x >> 5;
    const int G = p.H / p.KV, groups = (G + GH - 1) / GH;
    const int kv = blockIdx.x / groups, hg = blockIdx.x - kv * groups, h0 = kv * G + hg * GH, nh = min(GH, G - hg * GH);
    float* q_s = reinterpret_cast<float*>(wr_sm);
    float* acc_s = q_s + GH * p.dim_p;
    TC* kn = reinterpret_cast<TC*>(acc_s + nw * GH * p.vdim_p);
    TC* vn = kn + p.dim_p;
    const int ks_t = p.dim_p + 16 / (int)sizeof(TC), vs_t = p.vdim_p + 16 / (int)sizeof(TC); // tile row strides: 16 bytes of padding
    TC* kt = vn + p.vdim_p + (size_t)warp * 32 * (ks_t + vs_t);
    TC* vt = kt + 32 * ks_t;
    const bool early = p.pos_ptr != nullptr; // decode step
    if (!early) pdl_wait();
    const int s = blockIdx.z, pos = (p.pos_ptr ? p.pos_ptr[0] : p.pos0) + s;
    if (pos < 0 || pos >= p.max_ctx) { // refused before anything is read or written (the same for every CTA)
        if (tid == 0 && p.status) atomicExch(p.status, LB_DEV_POS_RANGE);
        if (early) pdl_wait();
        return;
    }
    const float* row = p.proj + (size_t)s * p.ld;
    const int w0 = p.block > 0 ? pos / p.block * p.block : 0, n = pos - w0 + 1;
    const int per = ((n + p.splits - 1) / p.splits + 31) & ~31, used = (n + per - 1) / per; // rows per slice; slices that have rows
    if ((int)blockIdx.y >= used) return;
    const int r0 = w0 + blockIdx.y * per, r1 = min(r0 + per, pos + 1); // this CTA's rows
    const bool own = p.k_off >= 0; // the newest row is made here
    TC* kc = reinterpret_cast<TC*>(p.k_cache) + (size_t)kv * p.dim_p;
    TC* vc = reinterpret_cast<TC*>(p.v_cache) + (size_t)kv * p.vdim_p;
    const size_t ks = (size_t)p.KV * p.dim_p, vs = (size_t)p.KV * p.vdim_p;
    auto stage = [&](int b) { // rows b .. b + 31 (those past the slice repeat its last one; the newest row's place is not used)
        constexpr int E = 16 / (int)sizeof(TC);
        const int kq = p.dim_p / E, vq = p.vdim_p / E;
        for (int i = lane; i < 32 * kq; i += 32) {
            const int r = i / kq, c = i - r * kq;
            ms_cp16(smem_u32(kt + r * ks_t + c * E), kc + (size_t)min(b + r, r1 - 1) * ks + c * E);
        }
        for (int i = lane; i < 32 * vq; i += 32) {
            const int r = i / vq, c = i - r * vq;
            ms_cp16(smem_u32(vt + r * vs_t + c * E), vc + (size_t)min(b + r, r1 - 1) * vs + c * E);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (r0 + warp * 32 < r1) stage(r0 + warp * 32);
    wa_fill_angles(p, pos, A);
    __syncthreads();
    if (early) pdl_wait();
    for (int g = warp; g < GH; g += nw) {
        float* dst = q_s + g * p.dim_p;
        if (g < nh) wa_warp_rotate(row + p.q_off + (size_t)(h0 + g) * p.dim, dst, p.dim, p.rot_dims, A.ck, A.sk, p.scale);
        for (int i = lane; i < p.dim_p; i += 32)
            if (g >= nh || i >= p.dim) dst[i] = 0.f;
    }
    const bool has_new = own && pos < r1;
    if (has_new) {
        if (warp == nw - 1) wa_warp_rotate(row + p.k_off + (size_t)kv * p.dim, kn, p.dim, p.rot_dims, A.ck, A.sk, 1.f);
        if (warp == (nw > 1 ? nw - 2 : 0)) wa_warp_value(p, row + p.v_off + (size_t)kv * p.vdim, vn, A);
        for (int i = tid; i < p.dim_p; i += blockDim.x)
            if (i >= p.dim) kn[i] = wa_t<TC>::from(0.f);
        for (int i = tid; i < p.vdim_p; i += blockDim.x)
            if (i >= p.vdim) vn[i] = wa_t<TC>::from(0.f);
    }
    __syncthreads();
    if (has_new && hg == 0) { // one of the head groups appends the row
        for (int i = tid; i < p.dim_p; i += blockDim.x) kc[(size_t)pos * ks + i] = kn[i];
        for (int i = tid; i < p.vdim_p; i += blockDim.x) vc[(size_t)pos * vs + i] = vn[i];
    }
    pdl_launch_dependents();

    float m[GH], l[GH], acc[GH][2 * NV];
#pragma unroll
    for (int g = 0; g < GH; ++g) {
        m[g] = -1e30f;
        l[g] = 0.f;
#pragma unroll
        for (int i = 0; i < 2 * NV; ++i) acc[g][i] = 0.f;
    }
    for (int b = r0 + warp * 32; b < r1; b += nw * 32) {
        if (b != r0 + warp * 32) stage(b);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncwarp();
        const TC* kr = own && b + lane == pos ? kn : kt + lane * ks_t;
        float sc[GH];
#pragma unroll
        for (int g = 0; g < GH; ++g) sc[g] = 0.f;
#pragma unroll 4
        for (int d = 0; d < p.dim_p; d += 8) {
            float kf[8];
            wa_t<TC>::ld8(kr + d, kf);
#pragma unroll
            for (int g = 0; g < GH; ++g) {
                const float4 qa = *reinterpret_cast<const float4*>(q_s + g * p.dim_p + d), qb = *reinterpret_cast<const float4*>(q_s + g * p.dim_p + d + 4);
                sc[g] = fmaf(kf[0], qa.x, sc[g]);
                sc[g] = fmaf(kf[1], qa.y, sc[g]);
                sc[g] = fmaf(kf[2], qa.z, sc[g]);
                sc[g] = fmaf(kf[3], qa.w, sc[g]);
                sc[g] = fmaf(kf[4], qb.x, sc[g]);
                sc[g] = fmaf(kf[5], qb.y, sc[g]);
                sc[g] = fmaf(kf[6], qb.z, sc[g]);
                sc[g] = fmaf(kf[7], qb.w, sc[g]);
            }
        }
        const int cnt = min(32, r1 - b);
        float mx[GH], ps[GH];
#pragma unroll
        for (int g = 0; g < GH; ++g) mx[g] = lane < cnt ? sc[g] : -INFINITY;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1)
#pragma unroll
            for (int g = 0; g < GH; ++g) mx[g] = fmaxf(mx[g], __shfl_xor_sync(0xffffffffu, mx[g], o));
#pragma unroll
        for (int g = 0; g < GH; ++g) {
            const float mn = fmaxf(m[g], mx[g]), corr = expf(m[g] - mn), e = lane < cnt ? expf(sc[g] - mn) : 0.f;
            m[g] = mn;
            l[g] *= corr;
            ps[g] = e;
            pw[warp][lane][g] = e;
#pragma unroll
            for (int i = 0; i < 2 * NV; ++i) acc[g][i] *= corr;
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1)
#pragma unroll
            for (int g = 0; g < GH; ++g) ps[g] += __shfl_xor_sync(0xffffffffu, ps[g], o);
#pragma unroll
        for (int g = 0; g < GH; ++g) l[g] += ps[g];
        __syncwarp();
#pragma unroll 4
        for (int j = 0; j < cnt; ++j) {
            const TC* vr = own && b + j == pos ? vn : vt + j * vs_t;
            float2 vv[NV];
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const int d = 2 * lane + 64 * i;
                vv[i] = d < p.vdim_p ? wa_t<TC>::ld2(vr + d) : make_float2(0.f, 0.f);
            }
#pragma unroll
            for (int g = 0; g < GH; ++g) {
                const float e = pw[warp][j][g];
#pragma unroll
                for (int i = 0; i < NV; ++i) {
                    acc[g][2 * i] = fmaf(e, vv[i].x, acc[g][2 * i]);
                    acc[g][2 * i + 1] = fmaf(e, vv[i].y, acc[g][2 * i + 1]);
                }
            }
        }
        __syncwarp();
    }
    // warps of the CTA, in warp order
#pragma unroll
    for (int g = 0; g < GH; ++g) {
        if (lane == 0) { ml[warp][g][0] = m[g]; ml[warp][g][1] = l[g]; }
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int d = 2 * lane + 64 * i;
            if (d < p.vdim_p) *reinterpret_cast<float2*>(acc_s + (warp * GH + g) * p.vdim_p + d) = make_float2(acc[g][2 * i], acc[g][2 * i + 1]);
        }
    }
    __syncthreads();
    const int rec = p.vdim_p + 2;
    float* scr = p.scratch + ((size_t)blockIdx.x * p.splits) * GH * rec;
    if (used > 1) {
        float* mine = scr + (size_t)blockIdx.y * GH * rec;
        for (int i = tid; i < nh * p.vdim_p; i += blockDim.x) {
            const int g = i / p.vdim_p, d = i - g * p.vdim_p;
            float M = -1e30f, a = 0.f, L = 0.f;
            for (int w = 0; w < nw; ++w) M = fmaxf(M, ml[w][g][0]);
            for (int w = 0; w < nw; ++w) {
                const float f = expf(ml[w][g][0] - M);
                a = fmaf(f, acc_s[(w * GH + g) * p.vdim_p + d], a);
                L = fmaf(f, ml[w][g][1], L);
            }
            __stcg(mine + g * rec + d, a);
            if (d == 0) { __stcg(mine + g * rec + p.vdim_p, M); __stcg(mine + g * rec + p.vdim_p + 1, L); }
        }
        __threadfence();
        __syncthreads();
        if (tid == 0) {
            const uint32_t old = atomicAdd(p.counters + blockIdx.x, 1u);
            last_flag = old == (uint32_t)used - 1u;
            if (last_flag) p.counters[blockIdx.x] = 0u; // everybody has arrived: ready for the next launch
        }
        __syncthreads();
        if (!last_flag) return;
        __threadfence();
    }
    // the whole sum of each head (slices in order, or the warps of the only one), the sink, back-rotation by this position
    const int parts = used > 1 ? used : nw;
    if (tid < nh) {
        const int g = tid;
        float M = p.sink ? 0.f : -1e30f;
#pragma unroll 4
        for (int q = 0; q < parts; ++q) M = fmaxf(M, used > 1 ? __ldcg(scr + ((size_t)q * GH + g) * rec + p.vdim_p) : ml[q][g][0]);
        float L = p.sink ? expf(-M) : 0.f;
#pragma unroll 4
        for (int q = 0; q < parts; ++q) {
            const float f = expf((used > 1 ? __ldcg(scr + ((size_t)q * GH + g) * rec + p.vdim_p) : ml[q][g][0]) - M);
            L = fmaf(f, used > 1 ? __ldcg(scr + ((size_t)q * GH + g) * rec + p.vdim_p + 1) : ml[q][g][1], L);
            fw[q][g] = f;
        }
        for (int q = 0; q < parts; ++q) fw[q][g] /= L;
    }
    __syncthreads();
    for (int i = tid; i < nh * (p.vdim_p / 2); i += blockDim.x) {
        const int g = i / (p.vdim_p / 2), d = 2 * (i - g * (p.vdim_p / 2));
        if (d >= p.vdim) continue;
        float u = 0.f, v = 0.f;
        if (used > 1) {
#pragma unroll 8
            for (int q = 0; q < parts; ++q) {
                const float2 x = __ldcg(reinterpret_cast<const float2*>(scr + ((size_t)q * GH + g) * rec + d));
                u = fmaf(fw[q][g], x.x, u);
                v = fmaf(fw[q][g], x.y, v);
            }
        } else {
            for (int q = 0; q < parts; ++q) {
                u = fmaf(fw[q][g], acc_s[(q * GH + g) * p.vdim_p + d], u);
                v = fmaf(fw[q][g], acc_s[(q * GH + g) * p.vdim_p + d + 1], v);
            }
        }
        if (p.freq_v) {
            const float c = A.cv[d / 2], sn = A.sv[d / 2], a = u * c + v * sn;
            v = v * c - u * sn;
            u = a;
        }
        const int o = (h0 + g) * p.vdim + d;
        if (!p.cat) {
            p.out[o] = u;
            if (d + 1 < p.vdim) p.out[o + 1] = v;
        } else {
            TC* dst = reinterpret_cast<TC*>(p.cat) + (size_t)s * p.cat_ld + o;
            dst[0] = wa_t<TC>::from(u);
            if (d + 1 < p.vdim) dst[1] = wa_t<TC>::from(v);
        }
    }
}
#define WR_KERNEL(name, TC, GH, NV)                                                                                      \
    extern "C" __global__ void __launch_bounds__(WR_MAX_WARPS * 32) name(const __grid_constant__ lb_wattn_params p) {        \
        wattn_rows_body<TC, GH, NV>(p);                                                                                  \
    }
WR_KERNEL(wattn_rows_b2n2, __nv_bfloat16, 2, 2)
WR_KERNEL(wattn_rows_b4n2, __nv_bfloat16, 4, 2)
WR_KERNEL(wattn_rows_b8n2, __nv_bfloat16, 8, 2)
WR_KERNEL(wattn_rows_b2n4, __nv_bfloat16, 2, 4)
WR_KERNEL(wattn_rows_b4n4, __nv_bfloat16, 4, 4)
WR_KERNEL(wattn_rows_b8n4, __nv_bfloat16, 8, 4)
WR_KERNEL(wattn_rows_f2n2, float, 2, 2)
WR_KERNEL(wattn_rows_f4n2, float, 4, 2)
WR_KERNEL(wattn_rows_f8n2, float, 8, 2)
WR_KERNEL(wattn_rows_f2n4, float, 2, 4)
WR_KERNEL(wattn_rows_f4n4, float, 4, 4)
WR_KERNEL(wattn_rows_f8n4, float, 8, 4)

// A prompt chunk: keys and values of every token into the cache, queries as two bf16 terms (their sum carries 16 bits) pre-scaled so
// that scores come out in log2 units.  One block per token; a layer without keys of its own has only queries.  grid T, block 256
template <typename TC>
__device__ __forceinline__ void wattn_prepare_body(const lb_wattn_params& p) {
    __shared__ wa_angles A;
    __shared__ float q_s[8][LB_WA_MAX_DIM];
    pdl_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, s = blockIdx.x, pos = p.pos0 + s;
    const float* row = p.proj + (size_t)s * p.ld;
    wa_fill_angles(p, pos, A);
    __syncthreads();
    const int nk = p.k_off >= 0 ? p.KV : 0, nq = p.qh ? p.H : 0;
    for (int r = warp; r < 2 * nk + nq; r += 8) {
        if (r < nk) wa_warp_rotate(row + p.k_off + (size_t)r * p.dim, reinterpret_cast<TC*>(p.k_cache) + ((size_t)pos * p.KV + r) * p.dim_p, p.dim, p.rot_dims, A.ck, A.sk, 1.f);
        else if (r < 2 * nk) wa_warp_value(p, row + p.v_off + (size_t)(r - nk) * p.vdim, reinterpret_cast<TC*>(p.v_cache) + ((size_t)pos * p.KV + r - nk) * p.vdim_p, A);
        else {
            const int h = r - 2 * nk;
            wa_warp_rotate(row + p.q_off + (size_t)h * p.dim, q_s[warp], p.dim, p.rot_dims, A.ck, A.sk, p.scale * 1.4426950408889634f);
            __syncwarp();
            const size_t o = ((size_t)s * p.H + h) * p.dim_p;
            for (int i = lane; i < p.dim_p; i += 32) {
                const float q = i < p.dim ? q_s[warp][i] : 0.f;
                const __nv_bfloat16 hi = __float2bfloat16_rn(q);
                reinterpret_cast<__nv_bfloat16*>(p.qh)[o + i] = hi;
                reinterpret_cast<__nv_bfloat16*>(p.ql)[o + i] = __float2bfloat16_rn(q - __bfloat162float(hi));
            }
            __syncwarp();
        }
    }
    pdl_launch_dependents();
}
extern "C" __global__ void __launch_bounds__(256) wattn_prepare_bf16(const __grid_constant__ lb_wattn_params p) { wattn_prepare_body<__nv_bfloat16>(p); }
extern "C" __global__ void __launch_bounds__(256) wattn_prepare_f32(const __grid_constant__ lb_wattn_params p) { wattn_prepare_body<float>(p); }

// ---- a prompt chunk on the tensor cores -----------------------------------------------------------------------------
// grid (ceil(T G / LB_WA_ROWS), KV), block LB_WA_THREADS.  Query row R of a KV head = (token R / G, head R % G).  S = Q K^T and O = P V as
// mma.sync m16n8k16 with Q and P in two bf16 terms, online soft-max in log2 units (the sink enters as a first score: 0, or the head's own), cache rows staged
// LB_WA_KV at a time from the first block start any row of the CTA sees.  NB: value features / 8 the accumulators hold.
// dynamic shared memory: qh | ql [ROWS][2 dim_p + 16 B], then two stages of K [KV][2 dim_p + 16] and V [KV][2 vdim_p + 16]
template <int NB>
__device__ __forceinline__ void wattn_chunk_body(const lb_wattn_params& p) {
    extern __shared__ __align__(16) unsigned char wc_sm[];
    const int t = threadIdx.x, lane = t & 31, warp = t >> 5, fg = lane >> 2, ft = lane & 3;
    const int kv = blockIdx.y, G = p.H / p.KV, R0 = blockIdx.x * LB_WA_ROWS, n_rows = p.T * G;
    const int qst = 2 * p.dim_p + 16, vst = 2 * p.vdim_p + 16, q16 = p.dim_p / 8, v16 = p.vdim_p / 8;
    unsigned char* qh_s = wc_sm;
    unsigned char* ql_s = qh_s + LB_WA_ROWS * qst;
    unsigned char* kv_s = ql_s + LB_WA_ROWS * qst;
    const int stage_bytes = LB_WA_KV * (qst + vst);
    pdl_wait();
    for (int i = t; i < LB_WA_ROWS * q16; i += LB_WA_THREADS) { // rows past the chunk repeat the last one; they are never stored
        const int r = i / q16, c = i - r * q16, R = min(R0 + r, n_rows - 1), s = R / G;
        const size_t src = ((size_t)s * p.H + kv * G + (R - s * G)) * p.dim_p + c * 8;
        ms_cp16(smem_u32(qh_s + r * qst + c * 16), p.qh + src);
        ms_cp16(smem_u32(ql_s + r * qst + c * 16), p.ql + src);
    }
    const int s_first = R0 / G, s_last = min(R0 + LB_WA_ROWS - 1, n_rows - 1) / G;
    const int first_key = p.block > 0 ? (p.pos0 + s_first) / p.block * p.block : 0, last_key = p.pos0 + s_last;
    const int n_blocks = (last_key - first_key) / LB_WA_KV + 1;
    const int own_p = p.dim_p - p.tail_p, own16 = own_p / 8; // of a key: what the head has of its own
    const unsigned char* kbase = reinterpret_cast<const unsigned char*>(p.k_cache) + (size_t)kv * own_p * 2;
    const unsigned char* tbase = reinterpret_cast<const unsigned char*>(p.k_tail);
    const unsigned char* vbase = reinterpret_cast<const unsigned char*>(p.v_cache) + (size_t)kv * p.vdim_p * 2;
    const size_t krow = (size_t)p.KV * own_p * 2, vrow = (size_t)p.KV * p.vdim_p * 2, trow = (size_t)p.tail_ld * 2;
    auto stage = [&](int b) { // rows past the last one repeat it (finite values; masked below)
        unsigned char* dst = kv_s + (b & 1) * stage_bytes;
        for (int i = t; i < LB_WA_KV * (q16 + v16); i += LB_WA_THREADS) {
            const int r = i / (q16 + v16), c = i - r * (q16 + v16);
            const size_t row = (size_t)min(first_key + b * LB_WA_KV + r, last_key);
            if (c < own16) ms_cp16(smem_u32(dst + r * qst + c * 16), kbase + row * krow + c * 16);
            else if (c < q16) ms_cp16(smem_u32(dst + r * qst + c * 16), tbase + row * trow + (c - own16) * 16);
            else ms_cp16(smem_u32(dst + LB_WA_KV * qst + r * vst + (c - q16) * 16), vbase + row * vrow + (c - q16) * 16);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(0);
    int lim[2], low[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        lim[i] = p.pos0 + min(R0 + warp * 16 + fg + 8 * i, n_rows - 1) / G;
        low[i] = p.block > 0 ? lim[i] / p.block * p.block : 0;
    }
    const int w_last = p.pos0 + min(R0 + warp * 16 + 15, n_rows - 1) / G;
    const int w_pos = p.pos0 + min(R0 + warp * 16, n_rows - 1) / G, w_first = p.block > 0 ? w_pos / p.block * p.block : 0;
    float m_run[2], l_run[2], acc[NB][4];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        m_run[i] = !p.sink ? -1e30f : p.sink_w ? bf16_bits_to_f32(p.sink_w[kv * G + min(R0 + warp * 16 + fg + 8 * i, n_rows - 1) % G]) * 1.4426950408889634f : 0.f;
        l_run[i] = p.sink ? 1.f : 0.f;
    }
#pragma unroll
    for (int nb = 0; nb < NB; ++nb) acc[nb][0] = acc[nb][1] = acc[nb][2] = acc[nb][3] = 0.f;
    const uint32_t a_off = (warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * qst + (lane >> 4) * 16;
    const uint32_t qh_lane = smem_u32(qh_s) + a_off, ql_lane = smem_u32(ql_s) + a_off;
    const uint32_t k_off = ((lane & 7) + ((lane >> 4) << 3)) * qst + ((lane >> 3) & 1) * 16;
    const uint32_t v_off = ((lane & 7) + ((lane >> 3) & 1) * 8) * vst + (lane >> 4) * 16;
    const int nkc = p.dim_p / 16, nvb = p.vdim_p / 8;

    for (int b = 0; b < n_blocks; ++b) {
        if (b + 1 < n_blocks) {
            stage(b + 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const int key0 = first_key + b * LB_WA_KV;
        if (key0 <= w_last && key0 + LB_WA_KV > w_first) {
            const uint32_t k_addr = smem_u32(kv_s + (b & 1) * stage_bytes), v_addr = k_addr + LB_WA_KV * qst;
            float sc[4][4];
#pragma unroll
            for (int j = 0; j < 4; ++j) sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.f;
#pragma unroll 4
            for (int c = 0; c < nkc; ++c) {
                uint32_t h0, h1, h2, h3, l0, l1, l2, l3;
                ms_ldsm(qh_lane + c * 32, h0, h1, h2, h3);
                ms_ldsm(ql_lane + c * 32, l0, l1, l2, l3);
#pragma unroll
                for (int jj = 0; jj < 2; ++jj) {
                    uint32_t b00, b01, b10, b11;
                    ms_ldsm(k_addr + k_off + jj * 16 * qst + c * 32, b00, b01, b10, b11);
                    ms_mma(sc[2 * jj], h0, h1, h2, h3, b00, b01);
                    ms_mma(sc[2 * jj], l0, l1, l2, l3, b00, b01);
                    ms_mma(sc[2 * jj + 1], h0, h1, h2, h3, b10, b11);
                    ms_mma(sc[2 * jj + 1], l0, l1, l2, l3, b10, b11);
                }
            }
            float corr[2];
            uint32_t ph[4][2], pl[4][2];
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                float mx = -INFINITY;
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const int r0 = key0 + 8 * j + 2 * ft;
                    if (r0 > lim[i] || r0 < low[i]) sc[j][2 * i] = -INFINITY;
                    if (r0 + 1 > lim[i] || r0 + 1 < low[i]) sc[j][2 * i + 1] = -INFINITY;
                    mx = fmaxf(mx, fmaxf(sc[j][2 * i], sc[j][2 * i + 1]));
                }
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
                const float m_new = fmaxf(m_run[i], mx); // never -inf: m_run starts finite
                corr[i] = exp2f(m_run[i] - m_new);
                float ps = 0.f;
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const float p0 = exp2f(sc[j][2 * i] - m_new), p1 = exp2f(sc[j][2 * i + 1] - m_new);
                    ps += p0 + p1;
                    ms_split(p0, p1, ph[j][i], pl[j][i]);
                }
                ps += __shfl_xor_sync(0xffffffffu, ps, 1);
                ps += __shfl_xor_sync(0xffffffffu, ps, 2);
                l_run[i] = fmaf(l_run[i], corr[i], ps);
                m_run[i] = m_new;
            }
#pragma unroll
            for (int nb = 0; nb < NB; nb += 2) {
                if (nb < nvb) {
                    acc[nb][0] *= corr[0]; acc[nb][1] *= corr[0]; acc[nb][2] *= corr[1]; acc[nb][3] *= corr[1];
                    acc[nb + 1][0] *= corr[0]; acc[nb + 1][1] *= corr[0]; acc[nb + 1][2] *= corr[1]; acc[nb + 1][3] *= corr[1];
#pragma unroll
                    for (int kk = 0; kk < 2; ++kk) {
                        uint32_t v0, v1, v2, v3;
                        ms_ldsm_t(v_addr + v_off + kk * 16 * vst + nb * 16, v0, v1, v2, v3);
                        ms_mma(acc[nb], ph[2 * kk][0], ph[2 * kk][1], ph[2 * kk + 1][0], ph[2 * kk + 1][1], v0, v1);
                        ms_mma(acc[nb], pl[2 * kk][0], pl[2 * kk][1], pl[2 * kk + 1][0], pl[2 * kk + 1][1], v0, v1);
                        ms_mma(acc[nb + 1], ph[2 * kk][0], ph[2 * kk][1], ph[2 * kk + 1][0], ph[2 * kk + 1][1], v2, v3);
                        ms_mma(acc[nb + 1], pl[2 * kk][0], pl[2 * kk][1], pl[2 * kk + 1][0], pl[2 * kk + 1][1], v2, v3);
                    }
                }
            }
        }
        __syncthreads(); // every warp is done with this stage before block b+2 overwrites it
    }
    pdl_launch_dependents();
    // lane (fg, ft) holds features 8 nb + 2 ft, +1 of rows fg and fg + 8: a value pair turns back by its token's position
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int R = R0 + warp * 16 + fg + 8 * i;
        if (R >= n_rows) continue;
        const int s = R / G, h = kv * G + (R - s * G);
        const float inv = 1.0f / l_run[i];
        __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(p.cat) + (size_t)s * p.cat_ld + (size_t)h * p.vdim;
#pragma unroll
        for (int nb = 0; nb < NB; ++nb) {
            const int d = 8 * nb + 2 * ft;
            if (d >= p.vdim) continue;
            float u = acc[nb][2 * i] * inv, v = acc[nb][2 * i + 1] * inv;
            if (p.freq_v) {
                float c, sn;
                wa_angle(p.freq_v[d / 2], lim[i], c, sn);
                const float a = u * c + v * sn;
                v = v * c - u * sn;
                u = a;
            }
            dst[d] = __float2bfloat16_rn(u);
            if (d + 1 < p.vdim) dst[d + 1] = __float2bfloat16_rn(v);
        }
    }
}
extern "C" __global__ void __launch_bounds__(LB_WA_THREADS) wattn_chunk_64(const __grid_constant__ lb_wattn_params p) { wattn_chunk_body<8>(p); }
extern "C" __global__ void __launch_bounds__(LB_WA_THREADS) wattn_chunk_128(const __grid_constant__ lb_wattn_params p) { wattn_chunk_body<16>(p); }
extern "C" __global__ void __launch_bounds__(LB_WA_THREADS) wattn_chunk_256(const __grid_constant__ lb_wattn_params p) { wattn_chunk_body<32>(p); }
