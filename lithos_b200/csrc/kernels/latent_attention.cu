// Attention over a cached latent: a position is cached as one row [c | kr], c the normed latent, kr one rotated key part shared by all heads.
//   key of head h = [W_uk,h c | kr],  value = W_uv,h c,  weight of key j at position i = exp(s_ij) / (exp(sink_h) + sum exp(s)), s = scale q.k
// Two ways to compute it.  Absorbed: q.(W_uk c) = (W_uk^T q).c, so queries become rows of the cache's shape, the weighted sum of latents passes
// W_uv once; nothing is made per cached position (decode, short portions, fp32).  Expanded: a product makes every position's keys and values
// for the tensor-core kernel of window_attention.cu (prompt chunks).  Scores, weights and sums are fp32; angles are reduced in double.
//   lat_query_*    absorbed: new cache rows; queries (W_uk^T q | rotated part) * scale
//   lat_rows_bf16  absorbed: queries x a slice of the cache rows on the tensor cores;  lat_rows_f32 the same in fp32
//   lat_out_*      absorbed: slices merged, the sink, W_uv
//   lat_prepare_*  expanded: new cache rows; queries as two bf16 terms
#include "mma_sync.cuh"
#include "rotate.cuh"

#define LA_THREADS 256

// the cache row of token s at position pos, by one block
template <typename TC>
__device__ __forceinline__ void la_cache_row(const lb_latent_params& p, int s, int pos, float* red) {
    const int t = threadIdx.x;
    const float *c = p.proj + (size_t)s * p.ld + p.kv_off, *k = c + p.rank;
    TC* row = reinterpret_cast<TC*>(p.cache) + (size_t)pos * (p.rank_p + p.rot_p);
    float ss = 0.f;
    for (int i = t; i < p.rank; i += blockDim.x) ss += c[i] * c[i];
    const float r = 1.0f / sqrtf(block_sum(ss, red) / (float)p.rank + p.eps);
    for (int i = t; i < p.rank; i += blockDim.x) row[i] = wa_t<TC>::from(c[i] * r * bf16_bits_to_f32(p.c_norm[i]));
    for (int i = t; i < p.rot / 2; i += blockDim.x) {
        float cs, sn;
        wa_angle(p.freq[i], pos, cs, sn);
        const float u = k[2 * i], v = k[2 * i + 1];
        row[p.rank_p + 2 * i] = wa_t<TC>::from((u * cs - v * sn) * p.rot_mul);
        row[p.rank_p + 2 * i + 1] = wa_t<TC>::from((v * cs + u * sn) * p.rot_mul);
    }
}

// grid (H + 1, ceil(rank_p / 128), ceil(T / LB_LA_TOKENS)), block 256; block column H makes the cache rows.  Thread (8 latent columns, one of 16
// parts of the head's features); the first eight rows of its weights come in before the wait.  dynamic shared memory: [16][128] fp32
template <typename TC>
__device__ __forceinline__ void lat_query_body(const lb_latent_params& p) {
    __shared__ float red[40], q_s[256 + LB_LA_MAX_ROT];
    __shared__ __align__(16) float sum_s[16][128 + 4];
    const int h = blockIdx.x, t = threadIdx.x, cg = t & 15, part = t >> 4, col = blockIdx.y * 128 + cg * 8;
    const int t0 = blockIdx.z * LB_LA_TOKENS, t1 = min(p.T, t0 + LB_LA_TOKENS), pos0 = p.pos_ptr ? p.pos_ptr[0] : p.pos0;
    if (pos0 < 0 || pos0 + p.T > p.max_ctx) { // refused before anything is read or written (the same for every CTA)
        if (t == 0 && p.status) atomicExch(p.status, LB_DEV_POS_RANGE);
        pdl_wait();
        return;
    }
    if (h == p.H) {
        pdl_wait();
        if (blockIdx.y == 0)
            for (int s = t0; s < t1; ++s) la_cache_row<TC>(p, s, pos0 + s, red);
        pdl_launch_dependents();
        return;
    }
    const bool live = col < p.rank_p; // rank_p is a multiple of 64, so a thread's eight columns exist or do not
    const uint16_t* w = p.uk + (size_t)h * p.dim * p.rank_p + col;
    uint4 pre[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) pre[i] = live && part + 16 * i < p.dim ? __ldg(reinterpret_cast<const uint4*>(w + (size_t)(part + 16 * i) * p.rank_p)) : make_uint4(0u, 0u, 0u, 0u);
    pdl_wait();
    const int qd = p.dim + p.rot, ld_c = p.rank_p + p.rot_p;
    for (int s = t0; s < t1; ++s) {
        const float* q = p.q + ((size_t)s * p.H + h) * qd;
        __syncthreads();
        for (int i = t; i < qd; i += LA_THREADS) q_s[i] = q[i];
        __syncthreads();
        float acc[8] = {};
        auto add = [&](const uint4& u, float x) {
            const uint32_t v[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                acc[2 * e] = fmaf(__uint_as_float(v[e] << 16), x, acc[2 * e]);
                acc[2 * e + 1] = fmaf(__uint_as_float(v[e] & 0xffff0000u), x, acc[2 * e + 1]);
            }
        };
#pragma unroll
        for (int i = 0; i < 8; ++i)
            if (part + 16 * i < p.dim) add(pre[i], q_s[part + 16 * i]);
        if (live)
            for (int d = part + 128; d < p.dim; d += 16) add(__ldg(reinterpret_cast<const uint4*>(w + (size_t)d * p.rank_p)), q_s[d]);
#pragma unroll
        for (int e = 0; e < 8; ++e) sum_s[part][cg * 8 + e] = acc[e];
        __syncthreads();
        float* out = p.ql + ((size_t)s * p.H + h) * ld_c;
        if (t < 128 && blockIdx.y * 128 + t < p.rank_p) {
            float a = 0.f;
#pragma unroll
            for (int k = 0; k < 16; ++k) a += sum_s[k][t];
            out[blockIdx.y * 128 + t] = a * p.scale;
        }
        if (blockIdx.y == 0)
            for (int i = t; i < p.rot_p / 2; i += LA_THREADS) {
                float a = 0.f, b = 0.f;
                if (2 * i < p.rot) {
                    float cs, sn;
                    wa_angle(p.freq[i], pos0 + s, cs, sn);
                    const float u = q_s[p.dim + 2 * i], v = q_s[p.dim + 2 * i + 1], m = p.rot_mul * p.scale;
                    a = (u * cs - v * sn) * m;
                    b = (v * cs + u * sn) * m;
                }
                out[p.rank_p + 2 * i] = a;
                out[p.rank_p + 2 * i + 1] = b;
            }
    }
    pdl_launch_dependents();
}
extern "C" __global__ void __launch_bounds__(LA_THREADS) lat_query_bf16(const __grid_constant__ lb_latent_params p) { lat_query_body<__nv_bfloat16>(p); }
extern "C" __global__ void __launch_bounds__(LA_THREADS) lat_query_f32(const __grid_constant__ lb_latent_params p) { lat_query_body<float>(p); }

// slices of positions 0 .. last: rows per slice, a multiple of the staged block
__device__ __forceinline__ int la_slice(int n, int splits) { return ((n + splits - 1) / splits + LB_LA_KEYS - 1) / LB_LA_KEYS * LB_LA_KEYS; }

// grid (ceil(T H / 16), splits), block 128.  Row R of the launch = (token R / H, head R % H); a CTA has 16 of them and one slice of the cache.
// A block of 64 cache rows serves as keys (all of it) and as values (its latent columns).  Scores: warp w has the block's rows 16 w ..; weighted
// sum: warp w has a quarter of the latent columns.  Queries and weights enter as two bf16 terms; soft-max in log2 units.  The first block's old
// rows are asked for before the wait for the queries and the newest rows.
// dynamic shared memory: query terms [2][16][2 ld_c + 16 B], weight terms [2][16][144 B], staged blocks [stages][64][2 ld_c + 16 B]
#define LR_PST 144
template <int NB> // latent columns / 32 the accumulators hold, rounded up to an even number of 8-column tiles per warp
__device__ __forceinline__ void lat_rows_body(const lb_latent_params& p) {
    extern __shared__ __align__(16) unsigned char lr_sm[];
    __shared__ float mx_s[4][16], sum_s[4][16];
    const int t = threadIdx.x, lane = t & 31, warp = t >> 5, fg = lane >> 2, ft = lane & 3;
    const int R0 = blockIdx.x * 16, n_rows = p.T * p.H, ld_c = p.rank_p + p.rot_p, st = 2 * ld_c + 16, c16 = ld_c / 8;
    const int pos0 = p.pos_ptr ? p.pos_ptr[0] : p.pos0, n = pos0 + p.T, per = la_slice(n, p.splits), used = (n + per - 1) / per;
    if (pos0 < 0 || n > p.max_ctx || (int)blockIdx.y >= used) {
        pdl_wait();
        return;
    }
    const int k0 = blockIdx.y * per, k1 = min(n, k0 + per); // this CTA's cache rows
    unsigned char *qh_s = lr_sm, *ql_s = qh_s + 16 * st, *ph_s = ql_s + 16 * st, *pl_s = ph_s + 16 * LR_PST, *kv_s = pl_s + 16 * LR_PST;
    const unsigned char* cache = reinterpret_cast<const unsigned char*>(p.cache);
    // rows of a block with old <= (row >= pos0) <= new...: rows before pos0 exist since an earlier step
    auto stage = [&](int b, bool old_rows, bool new_rows) {
        unsigned char* dst = kv_s + (p.stages > 1 ? b & 1 : 0) * (LB_LA_KEYS * st);
        for (int r = t >> 3; r < LB_LA_KEYS; r += 16) { // eight threads per row
            const int row = min(k0 + b * LB_LA_KEYS + r, k1 - 1);
            if (!(row < pos0 ? old_rows : new_rows)) continue;
            const unsigned char* src = cache + (size_t)row * ld_c * 2;
            const uint32_t to = smem_u32(dst + r * st);
#pragma unroll 3
            for (int c = t & 7; c < c16; c += 8) ms_cp16(to + c * 16, src + c * 16);
        }
    };
    stage(0, true, false);
    pdl_wait();
    stage(0, false, true);
    asm volatile("cp.async.commit_group;" ::: "memory");
    { // rows past the last one repeat it; they are not stored.  Eight threads per row, nine quads of each in flight
        const int r = t >> 3;
        const float4* q = reinterpret_cast<const float4*>(p.ql + (size_t)min(R0 + r, n_rows - 1) * ld_c);
        for (int c0 = t & 7; c0 < ld_c / 4; c0 += 72) {
            float4 v[9];
#pragma unroll
            for (int k = 0; k < 9; ++k) v[k] = c0 + 8 * k < ld_c / 4 ? q[c0 + 8 * k] : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int k = 0; k < 9; ++k) {
                if (c0 + 8 * k >= ld_c / 4) continue;
                uint2 hi, lo;
                ms_split(v[k].x * 1.4426950408889634f, v[k].y * 1.4426950408889634f, hi.x, lo.x);
                ms_split(v[k].z * 1.4426950408889634f, v[k].w * 1.4426950408889634f, hi.y, lo.y);
                *reinterpret_cast<uint2*>(qh_s + r * st + (c0 + 8 * k) * 8) = hi;
                *reinterpret_cast<uint2*>(ql_s + r * st + (c0 + 8 * k) * 8) = lo;
            }
        }
    }
    int lim[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) lim[r] = pos0 + min(R0 + fg + 8 * r, n_rows - 1) / p.H;
    float m_run[2] = {-1e30f, -1e30f}, l_run[2] = {0.f, 0.f}, acc[NB][4];
#pragma unroll
    for (int j = 0; j < NB; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
    const uint32_t a_off = ((lane & 7) + ((lane >> 3) & 1) * 8) * st + (lane >> 4) * 16;
    const uint32_t qh_lane = smem_u32(qh_s) + a_off, ql_lane = smem_u32(ql_s) + a_off;
    const uint32_t p_off = ((lane & 7) + ((lane >> 3) & 1) * 8) * LR_PST + (lane >> 4) * 16;
    const uint32_t ph_lane = smem_u32(ph_s) + p_off, pl_lane = smem_u32(pl_s) + p_off;
    const uint32_t k_off = (warp * 16 + (lane & 7) + ((lane >> 4) << 3)) * st + ((lane >> 3) & 1) * 16;
    const int cols = p.rank_p / 4; // latent columns of a warp, a multiple of 16
    const uint32_t v_off = ((lane & 7) + ((lane >> 3) & 1) * 8) * st + (lane >> 4) * 16 + warp * cols * 2;
    const int n_blk = (k1 - k0 + LB_LA_KEYS - 1) / LB_LA_KEYS, nkc = ld_c / 16;
    for (int b = 0; b < n_blk; ++b) {
        if (p.stages > 1 && b + 1 < n_blk) {
            stage(b + 1, true, true);
            asm volatile("cp.async.commit_group;\n\tcp.async.wait_group 1;" ::: "memory");
        } else asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        const uint32_t blk = smem_u32(kv_s) + (p.stages > 1 ? b & 1 : 0) * (LB_LA_KEYS * st);
        float sc[2][4] = {}, sl[2][4] = {};
#pragma unroll 4
        for (int c = 0; c < nkc; ++c) {
            uint32_t h0, h1, h2, h3, l0, l1, l2, l3, b0, b1, b2, b3;
            ms_ldsm(qh_lane + c * 32, h0, h1, h2, h3);
            ms_ldsm(ql_lane + c * 32, l0, l1, l2, l3);
            ms_ldsm(blk + k_off + c * 32, b0, b1, b2, b3);
            ms_mma(sc[0], h0, h1, h2, h3, b0, b1);
            ms_mma(sc[1], h0, h1, h2, h3, b2, b3);
            ms_mma(sl[0], l0, l1, l2, l3, b0, b1);
            ms_mma(sl[1], l0, l1, l2, l3, b2, b3);
        }
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) sc[j][e] += sl[j][e];
        const int key0 = k0 + b * LB_LA_KEYS + warp * 16 + 2 * ft;
#pragma unroll
        for (int r = 0; r < 2; ++r) { // maxima of the warp's 16 keys
            float mx = -INFINITY;
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    float& v = sc[j][2 * r + e];
                    if (key0 + 8 * j + e > lim[r] || key0 + 8 * j + e >= k1) v = -INFINITY;
                    mx = fmaxf(mx, v);
                }
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
            if (ft == 0) mx_s[warp][fg + 8 * r] = mx;
        }
        __syncthreads();
        float corr[2];
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int row = fg + 8 * r;
            const float m_new = fmaxf(m_run[r], fmaxf(fmaxf(mx_s[0][row], mx_s[1][row]), fmaxf(mx_s[2][row], mx_s[3][row])));
            corr[r] = exp2f(m_run[r] - m_new);
            m_run[r] = m_new;
            float ps = 0.f;
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const float e0 = exp2f(sc[j][2 * r] - m_new), e1 = exp2f(sc[j][2 * r + 1] - m_new);
                ps += e0 + e1;
                uint32_t hi, lo;
                ms_split(e0, e1, hi, lo);
                const int o = row * LR_PST + (warp * 16 + 8 * j + 2 * ft) * 2;
                *reinterpret_cast<uint32_t*>(ph_s + o) = hi;
                *reinterpret_cast<uint32_t*>(pl_s + o) = lo;
            }
            ps += __shfl_xor_sync(0xffffffffu, ps, 1);
            ps += __shfl_xor_sync(0xffffffffu, ps, 2);
            l_run[r] = fmaf(l_run[r], corr[r], ps); // this warp's keys
        }
        __syncthreads();
        uint32_t ph[4][4], pl[4][4];
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
            ms_ldsm(ph_lane + kk * 32, ph[kk][0], ph[kk][1], ph[kk][2], ph[kk][3]);
            ms_ldsm(pl_lane + kk * 32, pl[kk][0], pl[kk][1], pl[kk][2], pl[kk][3]);
        }
#pragma unroll
        for (int nb = 0; nb < NB; nb += 2) {
            if (nb * 8 >= cols) continue;
            acc[nb][0] *= corr[0]; acc[nb][1] *= corr[0]; acc[nb][2] *= corr[1]; acc[nb][3] *= corr[1];
            acc[nb + 1][0] *= corr[0]; acc[nb + 1][1] *= corr[0]; acc[nb + 1][2] *= corr[1]; acc[nb + 1][3] *= corr[1];
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) {
                uint32_t v0, v1, v2, v3;
                ms_ldsm_t(blk + v_off + kk * 16 * st + nb * 16, v0, v1, v2, v3);
                ms_mma(acc[nb], ph[kk][0], ph[kk][1], ph[kk][2], ph[kk][3], v0, v1);
                ms_mma(acc[nb], pl[kk][0], pl[kk][1], pl[kk][2], pl[kk][3], v0, v1);
                ms_mma(acc[nb + 1], ph[kk][0], ph[kk][1], ph[kk][2], ph[kk][3], v2, v3);
                ms_mma(acc[nb + 1], pl[kk][0], pl[kk][1], pl[kk][2], pl[kk][3], v2, v3);
            }
        }
        __syncthreads(); // everybody is done with this block, its maxima and weights
        if (p.stages == 1 && b + 1 < n_blk) {
            stage(b + 1, true, true);
            asm volatile("cp.async.commit_group;" ::: "memory");
        }
    }
    pdl_launch_dependents();
    if (ft == 0) { sum_s[warp][fg] = l_run[0]; sum_s[warp][fg + 8] = l_run[1]; }
    __syncthreads();
    const int rec = p.rank_p + 2;
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const int row = fg + 8 * r;
        if (R0 + row >= n_rows) continue;
        float* dst = p.part + ((size_t)(R0 + row) * p.splits + blockIdx.y) * rec;
#pragma unroll
        for (int nb = 0; nb < NB; ++nb) {
            if (nb * 8 >= cols) continue;
            *reinterpret_cast<float2*>(dst + warp * cols + 8 * nb + 2 * ft) = make_float2(acc[nb][2 * r], acc[nb][2 * r + 1]);
        }
        if (warp == 0 && ft == 0) {
            dst[p.rank_p] = m_run[r] > -1e29f ? m_run[r] * 0.6931471805599453f : -1e30f;
            dst[p.rank_p + 1] = (sum_s[0][row] + sum_s[1][row]) + (sum_s[2][row] + sum_s[3][row]);
        }
    }
}
extern "C" __global__ void __launch_bounds__(128) lat_rows_128(const __grid_constant__ lb_latent_params p) { lat_rows_body<4>(p); }
extern "C" __global__ void __launch_bounds__(128) lat_rows_256(const __grid_constant__ lb_latent_params p) { lat_rows_body<8>(p); }
extern "C" __global__ void __launch_bounds__(128) lat_rows_512(const __grid_constant__ lb_latent_params p) { lat_rows_body<16>(p); }

// fp32: grid (T * ceil(H / 8), splits), block 128: a token's eight heads and one slice.  A lane scores one of 32 staged cache rows for two heads
// of its warp; then threads own latent columns.  dynamic shared memory: queries [8][ld_c], staged rows [32][ld_c + 4]
extern "C" __global__ void __launch_bounds__(128) lat_rows_f32(const __grid_constant__ lb_latent_params p) {
    extern __shared__ __align__(16) float lf_sm[];
    __shared__ float w_s[8][32], corr_s[8];
    const int t = threadIdx.x, lane = t & 31, warp = t >> 5, hg = (p.H + 7) / 8, ld_c = p.rank_p + p.rot_p, kst = ld_c + 4;
    const int s = blockIdx.x / hg, h0 = (blockIdx.x - s * hg) * 8, nh = min(8, p.H - h0);
    float *q_s = lf_sm, *k_s = q_s + 8 * ld_c;
    pdl_wait();
    const int pos0 = p.pos_ptr ? p.pos_ptr[0] : p.pos0, n = pos0 + p.T, per = la_slice(n, p.splits), used = (n + per - 1) / per, pos = pos0 + s;
    if (pos0 < 0 || n > p.max_ctx || (int)blockIdx.y >= used) return;
    const int k0 = blockIdx.y * per, k1 = min(pos + 1, k0 + per);
    const float* cache = reinterpret_cast<const float*>(p.cache);
    for (int i = t; i < 8 * ld_c; i += 128) {
        const int g = i / ld_c;
        q_s[i] = g < nh ? p.ql[((size_t)s * p.H + h0 + g) * ld_c + (i - g * ld_c)] : 0.f;
    }
    float m[2] = {-1e30f, -1e30f}, l[2] = {0.f, 0.f}, acc[8][LB_LA_MAX_RANK / 128];
#pragma unroll
    for (int g = 0; g < 8; ++g)
#pragma unroll
        for (int i = 0; i < LB_LA_MAX_RANK / 128; ++i) acc[g][i] = 0.f;
    for (int b = k0; b < k1; b += 32) {
        const int cnt = min(32, k1 - b);
        __syncthreads();
        for (int i = t; i < cnt * (ld_c / 4); i += 128) {
            const int r = i / (ld_c / 4), c = i - r * (ld_c / 4);
            *reinterpret_cast<float4*>(k_s + r * kst + 4 * c) = *reinterpret_cast<const float4*>(cache + (size_t)(b + r) * ld_c + 4 * c);
        }
        __syncthreads();
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int g = 2 * warp + e;
            float sc = -INFINITY;
            if (lane < cnt) {
                float a0 = 0.f, a1 = 0.f;
                for (int d = 0; d < ld_c; d += 4) {
                    const float4 k = *reinterpret_cast<const float4*>(k_s + lane * kst + d), q = *reinterpret_cast<const float4*>(q_s + g * ld_c + d);
                    a0 = fmaf(k.x, q.x, a0);
                    a1 = fmaf(k.y, q.y, a1);
                    a0 = fmaf(k.z, q.z, a0);
                    a1 = fmaf(k.w, q.w, a1);
                }
                sc = a0 + a1;
            }
            float mx = sc;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float mn = fmaxf(m[e], mx), corr = expf(m[e] - mn), w = lane < cnt ? expf(sc - mn) : 0.f;
            m[e] = mn;
            l[e] = fmaf(l[e], corr, warp_sum(w));
            w_s[g][lane] = w;
            if (lane == 0) corr_s[g] = corr;
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < LB_LA_MAX_RANK / 128; ++i) {
            const int c = t + 128 * i;
            if (c >= p.rank_p) continue;
#pragma unroll
            for (int g = 0; g < 8; ++g) acc[g][i] *= corr_s[g];
            for (int j = 0; j < cnt; ++j) {
                const float v = k_s[j * kst + c];
#pragma unroll
                for (int g = 0; g < 8; ++g) acc[g][i] = fmaf(w_s[g][j], v, acc[g][i]);
            }
        }
    }
    pdl_launch_dependents();
    const int rec = p.rank_p + 2;
#pragma unroll
    for (int g = 0; g < 8; ++g) {
        if (g >= nh) continue;
        float* dst = p.part + (((size_t)s * p.H + h0 + g) * p.splits + blockIdx.y) * rec;
#pragma unroll
        for (int i = 0; i < LB_LA_MAX_RANK / 128; ++i)
            if (t + 128 * i < p.rank_p) dst[t + 128 * i] = acc[g][i];
    }
#pragma unroll
    for (int e = 0; e < 2; ++e)
        if (2 * warp + e < nh && lane == 0) {
            float* dst = p.part + (((size_t)s * p.H + h0 + 2 * warp + e) * p.splits + blockIdx.y) * rec;
            dst[p.rank_p] = m[e];
            dst[p.rank_p + 1] = l[e];
        }
}

// grid (H, ceil(vdim / 32), ceil(T / LB_LA_TOKENS)), block 256: the slices of a token's head merged in order, the sink, then 32 rows of W_uv:
// four per warp, a lane has eight (or, from rank_p 256, sixteen) columns of each, asked for before the wait
template <typename TC>
__device__ __forceinline__ void lat_out_body(const lb_latent_params& p) {
    __shared__ __align__(16) float o_s[LB_LA_MAX_RANK];
    __shared__ float f_s[LB_LA_MAX_SPLITS];
    const int h = blockIdx.x, t = threadIdx.x, lane = t & 31, warp = t >> 5, row0 = blockIdx.y * 32 + warp * 4;
    const int t0 = blockIdx.z * LB_LA_TOKENS, t1 = min(p.T, t0 + LB_LA_TOKENS);
    uint4 w[4][2];
#pragma unroll
    for (int r = 0; r < 4; ++r)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int c = 8 * (lane + 32 * e);
            w[r][e] = row0 + r < p.vdim && c < p.rank_p ? __ldg(reinterpret_cast<const uint4*>(p.uv + ((size_t)h * p.vdim + row0 + r) * p.rank_p + c)) : make_uint4(0u, 0u, 0u, 0u);
        }
    const float sink = p.sink ? bf16_bits_to_f32(p.sink[h]) : -1e30f;
    pdl_wait();
    const int pos0 = p.pos_ptr ? p.pos_ptr[0] : p.pos0, n = pos0 + p.T, per = la_slice(n, p.splits), used = (n + per - 1) / per, rec = p.rank_p + 2;
    if (pos0 < 0 || n > p.max_ctx) return;
    for (int s = t0; s < t1; ++s) {
        const float* part = p.part + ((size_t)s * p.H + h) * p.splits * rec;
        __syncthreads();
        if (warp == 0) {
            float m[LB_LA_MAX_SPLITS / 32], l[LB_LA_MAX_SPLITS / 32], M = sink;
#pragma unroll
            for (int i = 0; i < LB_LA_MAX_SPLITS / 32; ++i) {
                const int q = lane + 32 * i;
                m[i] = q < used ? part[(size_t)q * rec + p.rank_p] : -1e30f;
                l[i] = q < used ? part[(size_t)q * rec + p.rank_p + 1] : 0.f;
                M = fmaxf(M, m[i]);
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, o));
            float L = 0.f;
#pragma unroll
            for (int i = 0; i < LB_LA_MAX_SPLITS / 32; ++i) {
                m[i] = expf(m[i] - M);
                L = fmaf(m[i], l[i], L);
            }
            L = warp_sum(L) + (p.sink ? expf(sink - M) : 0.f);
#pragma unroll
            for (int i = 0; i < LB_LA_MAX_SPLITS / 32; ++i) f_s[lane + 32 * i] = m[i] / L;
        }
        __syncthreads();
        if (2 * t < p.rank_p) {
            float2 a = make_float2(0.f, 0.f);
#pragma unroll 16
            for (int q = 0; q < used; ++q) {
                const float2 v = *reinterpret_cast<const float2*>(part + (size_t)q * rec + 2 * t);
                a.x = fmaf(f_s[q], v.x, a.x);
                a.y = fmaf(f_s[q], v.y, a.y);
            }
            *reinterpret_cast<float2*>(o_s + 2 * t) = a;
        }
        __syncthreads();
        float sum[4];
#pragma unroll
        for (int r = 0; r < 4; ++r) {
            float a = 0.f;
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int c = 8 * (lane + 32 * e);
                if (c >= p.rank_p) continue;
                const float4 x = *reinterpret_cast<const float4*>(o_s + c), y = *reinterpret_cast<const float4*>(o_s + c + 4);
                const uint4 u = w[r][e];
                a = fmaf(__uint_as_float(u.x << 16), x.x, a);
                a = fmaf(__uint_as_float(u.x & 0xffff0000u), x.y, a);
                a = fmaf(__uint_as_float(u.y << 16), x.z, a);
                a = fmaf(__uint_as_float(u.y & 0xffff0000u), x.w, a);
                a = fmaf(__uint_as_float(u.z << 16), y.x, a);
                a = fmaf(__uint_as_float(u.z & 0xffff0000u), y.y, a);
                a = fmaf(__uint_as_float(u.w << 16), y.z, a);
                a = fmaf(__uint_as_float(u.w & 0xffff0000u), y.w, a);
            }
            sum[r] = warp_sum(a);
        }
        if (lane == 0)
#pragma unroll
            for (int r = 0; r < 4; ++r) {
                if (row0 + r >= p.vdim) continue;
                const int o = h * p.vdim + row0 + r;
                if (p.cat) reinterpret_cast<TC*>(p.cat)[(size_t)s * p.cat_ld + o] = wa_t<TC>::from(sum[r]);
                else p.out[o] = sum[r];
            }
    }
    pdl_launch_dependents();
}
extern "C" __global__ void __launch_bounds__(LA_THREADS) lat_out_bf16(const __grid_constant__ lb_latent_params p) { lat_out_body<__nv_bfloat16>(p); }
extern "C" __global__ void __launch_bounds__(LA_THREADS) lat_out_f32(const __grid_constant__ lb_latent_params p) { lat_out_body<float>(p); }

// expanded, bf16: a chunk's cache rows; queries [dim_p | rot_p] x scale x log2(e) as two bf16 terms (their sum carries 16 bits).  grid T, block 256
extern "C" __global__ void __launch_bounds__(LA_THREADS) lat_prepare(const __grid_constant__ lb_latent_params p) {
    __shared__ float red[40], cs[LB_LA_MAX_ROT / 2], sn[LB_LA_MAX_ROT / 2];
    const int s = blockIdx.x, pos = p.pos0 + s, t = threadIdx.x;
    pdl_wait();
    la_cache_row<__nv_bfloat16>(p, s, pos, red);
    const float mul = p.scale * 1.4426950408889634f;
    for (int i = t; i < p.rot / 2; i += LA_THREADS) {
        wa_angle(p.freq[i], pos, cs[i], sn[i]);
        cs[i] *= p.rot_mul;
        sn[i] *= p.rot_mul;
    }
    __syncthreads();
    const int kd = p.dim_p + p.rot_p, qd = p.dim + p.rot, pairs = kd / 2;
    const float* q = p.q + (size_t)s * p.H * qd;
    uint32_t *qh = reinterpret_cast<uint32_t*>(p.qh + (size_t)s * p.H * kd), *ql = reinterpret_cast<uint32_t*>(p.ql16 + (size_t)s * p.H * kd);
    for (int i = t; i < p.H * pairs; i += LA_THREADS) {
        const int h = i / pairs, d = 2 * (i - h * pairs);
        float u = 0.f, v = 0.f;
        if (d < p.dim_p) {
            if (d < p.dim) u = q[h * qd + d];
            if (d + 1 < p.dim) v = q[h * qd + d + 1];
        } else if (d - p.dim_p < p.rot) {
            const int r = d - p.dim_p;
            const float a = q[h * qd + p.dim + r], b = q[h * qd + p.dim + r + 1];
            u = a * cs[r / 2] - b * sn[r / 2];
            v = b * cs[r / 2] + a * sn[r / 2];
        }
        ms_split(u * mul, v * mul, qh[i], ql[i]);
    }
    pdl_launch_dependents();
}
