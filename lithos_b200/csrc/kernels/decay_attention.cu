// Linear attention whose state decays per key channel:  S <- diag(a_t) S + k_t v_t^T,  o_t = S^T q_t  per head, fp32 throughout.
//   HGRN2: f = l + (1 - l) sigmoid(z + b), a = f, k = 1 - f, q = silu(zq)
//   GLA:   a = sigmoid(W2 (W1 h) + b)^(1/tau), k = zk, q = dk^-1/2 zq
// A column j of a head's state needs only v_j, so a CTA owns a 32-column slab of one head and holds it in registers: thread (column,
// row quarter) has R rows of its column (4 R >= dk; rows past dk stay zero), the sum over rows is R local terms and two shuffles.
//   da_step_*   one token (decode): makes q, k, a of its head from the projections, state read and written once
//   da_inputs   a prompt chunk's q, k, a
//   da_scan_*   a prompt chunk through the recurrence, the state on chip for all of it
//   da_finish   per-head norm (and output gate) of the chunk's read-outs
#include "common.cuh"
#include "params.h"

#define DA_COLS 32
#define DA_THREADS 128

__device__ __forceinline__ float da_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float da_log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// q, k, a of channel ch (= head * dk + i); row: the token's projections, z2: GLA's second low-rank product
__device__ __forceinline__ void da_channel(const lb_decay_params2& p, const float* row, int ch, float z2, float& q, float& k, float& a) {
    const float zq = row[p.q_off + ch];
    const float b = bf16_bits_to_f32(p.bias[ch]);
    if (p.kind == LB_DA_HGRN2) {
        const float z = row[p.k_off + ch] + b, lo = bf16_bits_to_f32(p.lower[ch]);
        q = zq * da_sigmoid(zq);
        a = fmaf(1.0f - lo, da_sigmoid(z), lo);
        k = (1.0f - lo) * da_sigmoid(-z); // 1 - a without cancellation
    } else {
        q = zq * p.q_scale;
        k = row[p.k_off + ch];
        a = expf(da_log_sigmoid(z2 + b) * p.inv_tau);
    }
}
__device__ __forceinline__ float da_dot_rank(const uint16_t* w, const float* x, int rank) {
    float s = 0.f;
    for (int r = 0; r < rank; ++r) s = fmaf(bf16_bits_to_f32(w[r]), x[r], s);
    return s;
}

// grid (H, ceil(dv / 32)), block 128
template <int R>
__device__ __forceinline__ void da_step_body(const lb_decay_params2& p) {
    __shared__ float q_s[4 * R], k_s[4 * R], a_s[4 * R];
    const int h = blockIdx.x, t = threadIdx.x, q4 = t & 3, j = blockIdx.y * DA_COLS + (t >> 2);
    const bool live = j < p.dv;
    float* S = p.state + ((size_t)h * p.dk + (size_t)q4 * R) * p.dv + j;
    const int rows = min(R, p.dk - q4 * R);
    float s[R];
#pragma unroll
    for (int r = 0; r < R; ++r) s[r] = live && r < rows ? S[(size_t)r * p.dv] : 0.f; // written a whole step ago: needs no wait
    pdl_wait();
    for (int i = t; i < 4 * R; i += DA_THREADS) {
        float q = 0.f, k = 0.f, a = 0.f;
        if (i < p.dk) {
            const int ch = h * p.dk + i;
            const float z2 = p.kind == LB_DA_GLA ? da_dot_rank(p.a2 + (size_t)ch * p.rank, p.proj + p.a1_off, p.rank) : 0.f;
            da_channel(p, p.proj, ch, z2, q, k, a);
        }
        q_s[i] = q;
        k_s[i] = k;
        a_s[i] = a;
    }
    const float v = live ? p.proj[p.v_off + (size_t)h * p.dv + j] : 0.f;
    __syncthreads();
    pdl_launch_dependents();
    float o0 = 0.f, o1 = 0.f;
#pragma unroll
    for (int r = 0; r < R; r += 2) {
        s[r] = fmaf(a_s[q4 * R + r], s[r], k_s[q4 * R + r] * v);
        s[r + 1] = fmaf(a_s[q4 * R + r + 1], s[r + 1], k_s[q4 * R + r + 1] * v);
        o0 = fmaf(s[r], q_s[q4 * R + r], o0);
        o1 = fmaf(s[r + 1], q_s[q4 * R + r + 1], o1);
    }
#pragma unroll
    for (int r = 0; r < R; ++r)
        if (live && r < rows) S[(size_t)r * p.dv] = s[r];
    float o = o0 + o1;
    o += __shfl_xor_sync(0xffffffffu, o, 1);
    o += __shfl_xor_sync(0xffffffffu, o, 2);
    if (live && q4 == 0) p.o[(size_t)h * p.dv + j] = o;
}
extern "C" __global__ void __launch_bounds__(DA_THREADS) da_step_64(const __grid_constant__ lb_decay_params2 p) { da_step_body<16>(p); }
extern "C" __global__ void __launch_bounds__(DA_THREADS) da_step_128(const __grid_constant__ lb_decay_params2 p) { da_step_body<32>(p); }
extern "C" __global__ void __launch_bounds__(DA_THREADS) da_step_256(const __grid_constant__ lb_decay_params2 p) { da_step_body<64>(p); }

// q, k, a of a chunk, [T, H, dk_p] with zero padding.  grid (ceil(H dk_p / 256), ceil(T / 8)), block 256: a thread makes one channel of
// eight tokens, so a row of W2 is read once per eight tokens.  dynamic shared memory: [8][rank] fp32
extern "C" __global__ void __launch_bounds__(256) da_inputs(const __grid_constant__ lb_decay_params2 p) {
    extern __shared__ float a1_s[];
    pdl_wait();
    const int t0 = blockIdx.y * 8, nt = min(8, p.T - t0);
    if (p.kind == LB_DA_GLA)
        for (int i = threadIdx.x; i < 8 * p.rank; i += 256) {
            const int u = i / p.rank;
            a1_s[i] = u < nt ? p.proj[(size_t)(t0 + u) * p.ld + p.a1_off + (i - u * p.rank)] : 0.f;
        }
    __syncthreads();
    const int c = blockIdx.x * 256 + threadIdx.x;
    if (c < p.H * p.dk_p) {
        const int h = c / p.dk_p, i = c - h * p.dk_p, ch = h * p.dk + i;
        const bool live = i < p.dk;
        float z2[8] = {};
        if (live && p.kind == LB_DA_GLA)
            for (int r = 0; r < p.rank; ++r) {
                const float w = bf16_bits_to_f32(p.a2[(size_t)ch * p.rank + r]);
#pragma unroll
                for (int u = 0; u < 8; ++u) z2[u] = fmaf(w, a1_s[u * p.rank + r], z2[u]);
            }
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            if (u >= nt) break;
            float q = 0.f, k = 0.f, a = 0.f;
            if (live) da_channel(p, p.proj + (size_t)(t0 + u) * p.ld, ch, z2[u], q, k, a);
            const size_t o = (size_t)(t0 + u) * p.H * p.dk_p + c;
            p.q[o] = q;
            p.k[o] = k;
            p.a[o] = a;
        }
    }
    pdl_launch_dependents();
}

// grid (H, ceil(dv / 32)), block 128.  Operands of DA_U tokens at a time come DA_AHEAD stages ahead by cp.async (a row quarter of q, k, a
// is padded by 16 bytes so that the four quarters sit on different banks); one block barrier per DA_U tokens.
#define DA_U 4
#define DA_AHEAD 3
__device__ __forceinline__ void da_cp16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void da_cp4(void* dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
template <int R>
__device__ __forceinline__ void da_scan_body(const lb_decay_params2& p) {
    constexpr int QS = R + 4, VEC = 4 * QS, TOK = 3 * VEC + DA_COLS; // floats: a row quarter, a vector, a token's operands
    extern __shared__ __align__(16) float da_sm[];                   // [DA_AHEAD][DA_U][TOK]
    const int h = blockIdx.x, t = threadIdx.x, q4 = t & 3, jl = t >> 2, j = blockIdx.y * DA_COLS + jl;
    const bool live = j < p.dv;
    float* S = p.state + ((size_t)h * p.dk + (size_t)q4 * R) * p.dv + j;
    const int rows = min(R, p.dk - q4 * R);
    pdl_wait();
    const int n_st = (p.T + DA_U - 1) / DA_U;
    auto fetch = [&](int st) {
        float* dst = da_sm + (size_t)(st % DA_AHEAD) * (DA_U * TOK);
        constexpr int PIECES = 3 * R; // 16-byte pieces of q, k, a (4 R floats each)
        for (int i = t; i < DA_U * PIECES; i += DA_THREADS) {
            const int u = i / PIECES, c = i - u * PIECES, which = c / R, pc = c - which * R, tok = min(st * DA_U + u, p.T - 1);
            const float* src = (which == 0 ? p.q : which == 1 ? p.k : p.a) + ((size_t)tok * p.H + h) * (4 * R) + pc * 4;
            da_cp16(dst + u * TOK + which * VEC + (pc / (R / 4)) * QS + (pc % (R / 4)) * 4, src);
        }
        { // DA_U x 32 values: one per thread
            const int u = t >> 5, cc = t & 31, tok = min(st * DA_U + u, p.T - 1), col = min(blockIdx.y * DA_COLS + cc, p.dv - 1);
            da_cp4(dst + u * TOK + 3 * VEC + cc, p.proj + (size_t)tok * p.ld + p.v_off + (size_t)h * p.dv + col);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
#pragma unroll
    for (int st = 0; st < DA_AHEAD - 1; ++st) {
        if (st < n_st) fetch(st);
        else asm volatile("cp.async.commit_group;" ::: "memory");
    }
    float s[R];
#pragma unroll
    for (int r = 0; r < R; ++r) s[r] = live && r < rows ? S[(size_t)r * p.dv] : 0.f;
    for (int st = 0; st < n_st; ++st) {
        asm volatile("cp.async.wait_group %0;" ::"n"(DA_AHEAD - 2) : "memory");
        __syncthreads(); // everybody's pieces have landed, and everybody is done with the stage the next fetch fills
        if (st + DA_AHEAD - 1 < n_st) fetch(st + DA_AHEAD - 1);
        else asm volatile("cp.async.commit_group;" ::: "memory");
        const float* base = da_sm + (size_t)(st % DA_AHEAD) * (DA_U * TOK);
        float o[DA_U];
#pragma unroll
        for (int u = 0; u < DA_U; ++u) {
            const bool act = st * DA_U + u < p.T; // tokens past the chunk leave the state alone
            const float* tk = base + u * TOK;
            const float v = tk[3 * VEC + jl];
            const float4 *qv = reinterpret_cast<const float4*>(tk + q4 * QS), *kv = reinterpret_cast<const float4*>(tk + VEC + q4 * QS),
                         *av = reinterpret_cast<const float4*>(tk + 2 * VEC + q4 * QS);
            float o0 = 0.f, o1 = 0.f;
            if (act) {
#pragma unroll
                for (int c = 0; c < R / 4; ++c) {
                    const float4 q = qv[c], k = kv[c], a = av[c];
                    s[4 * c] = fmaf(a.x, s[4 * c], k.x * v);
                    s[4 * c + 1] = fmaf(a.y, s[4 * c + 1], k.y * v);
                    s[4 * c + 2] = fmaf(a.z, s[4 * c + 2], k.z * v);
                    s[4 * c + 3] = fmaf(a.w, s[4 * c + 3], k.w * v);
                    o0 = fmaf(s[4 * c], q.x, o0);
                    o1 = fmaf(s[4 * c + 1], q.y, o1);
                    o0 = fmaf(s[4 * c + 2], q.z, o0);
                    o1 = fmaf(s[4 * c + 3], q.w, o1);
                }
            }
            o[u] = o0 + o1;
        }
#pragma unroll
        for (int u = 0; u < DA_U; ++u) {
            o[u] += __shfl_xor_sync(0xffffffffu, o[u], 1);
            o[u] += __shfl_xor_sync(0xffffffffu, o[u], 2);
        }
        // lane q4 of a column stores token q4 of the four
        const float mine = q4 == 0 ? o[0] : q4 == 1 ? o[1] : q4 == 2 ? o[2] : o[3];
        const int tok = st * DA_U + q4;
        if (live && tok < p.T) p.o[(size_t)tok * p.H * p.dv + (size_t)h * p.dv + j] = mine;
    }
    pdl_launch_dependents();
#pragma unroll
    for (int r = 0; r < R; ++r)
        if (live && r < rows) S[(size_t)r * p.dv] = s[r];
}
static_assert(DA_U == 4 && DA_THREADS == 32 * DA_U, "one value per thread and stage; one token per lane of a column");
extern "C" __global__ void __launch_bounds__(DA_THREADS) da_scan_64(const __grid_constant__ lb_decay_params2 p) { da_scan_body<16>(p); }
extern "C" __global__ void __launch_bounds__(DA_THREADS) da_scan_128(const __grid_constant__ lb_decay_params2 p) { da_scan_body<32>(p); }
extern "C" __global__ void __launch_bounds__(DA_THREADS) da_scan_256(const __grid_constant__ lb_decay_params2 p) { da_scan_body<64>(p); }

// cat[t, h dv + i] = o / rms_head(o) * head_w[i] [ * silu(gate) ].  grid (T, ceil(H / 4)), block 128: one warp per (token, head)
extern "C" __global__ void __launch_bounds__(128) da_finish(const __grid_constant__ lb_decay_params2 p) {
    pdl_wait();
    const int s = blockIdx.x, h = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (h < p.H) {
        const float* o = p.o + ((size_t)s * p.H + h) * p.dv;
        float ss = 0.f;
        for (int i = lane; i < p.dv; i += 32) ss += o[i] * o[i];
        const float r = 1.0f / sqrtf(warp_sum(ss) / (float)p.dv + p.eps);
        for (int i = lane; i < p.dv; i += 32) {
            float v = o[i] * r * bf16_bits_to_f32(p.head_w[i]);
            if (p.g_off >= 0) {
                const float g = p.proj[(size_t)s * p.ld + p.g_off + (size_t)h * p.dv + i];
                v *= g * da_sigmoid(g);
            }
            const size_t d = (size_t)s * p.cat_ld + (size_t)h * p.dv + i;
            if (p.cat_f32) reinterpret_cast<float*>(p.cat)[d] = v;
            else reinterpret_cast<__nv_bfloat16*>(p.cat)[d] = __float2bfloat16_rn(v);
        }
    }
    pdl_launch_dependents();
}
