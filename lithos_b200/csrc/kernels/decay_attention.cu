// Linear attention whose state decays per key channel:  S <- diag(a_t) S + k_t v_t^T,  o_t = S^T q_t  per head, fp32 throughout.
//   HGRN2: f = l + (1 - l) sigmoid(z + b), a = f, k = 1 - f, q = silu(zq)
//   GLA:   a = sigmoid(W2 (W1 h) + b)^(1/tau), k = zk, q = dk^-1/2 zq
// A column j of a head's state needs only v_j, so a CTA owns a slab of columns of one head and holds it in registers: thread (column,
// row part) has R rows of its column (rows past dk stay zero), the sum over rows is local terms and a few shuffles.
//   da_step_*   one token (decode): makes q, k, a of its head from the projections, state read and written once
//   da_inputs   a prompt chunk's q, k, a
//   da_scan_*   a prompt chunk through the recurrence, the state on chip; a long chunk in two passes over segments of it, so that the
//               segments run side by side: da_local_* carries every segment from a zero state, da_scan_* starts each from its true state
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

// grid (H, ceil(dv / 32)), block 128; dynamic shared memory: GLA's W2 rows of the head, bf16 [dk][rank]
template <int R>
__device__ __forceinline__ void da_step_body(const lb_decay_params2& p) {
    extern __shared__ __align__(16) uint16_t a2_s[];
    __shared__ __align__(16) float q_s[4 * R], k_s[4 * R], a_s[4 * R], a1_s[256];
    const int h = blockIdx.x, t = threadIdx.x, q4 = t & 3, j = blockIdx.y * DA_COLS + (t >> 2);
    const bool live = j < p.dv, gla = p.kind == LB_DA_GLA;
    float* S = p.state + ((size_t)h * p.dk + (size_t)q4 * R) * p.dv + j;
    const int rows = min(R, p.dk - q4 * R);
    // constants, and the state (written a whole step ago), need no wait
    float s[R];
#pragma unroll
    for (int r = 0; r < R; ++r) s[r] = live && r < rows ? S[(size_t)r * p.dv] : 0.f;
    if (gla)
        for (int i = t; i < p.dk * p.rank; i += DA_THREADS) a2_s[i] = __ldg(p.a2 + (size_t)h * p.dk * p.rank + i);
    pdl_wait();
    const float v = live ? p.proj[p.v_off + (size_t)h * p.dv + j] : 0.f;
    if (gla) {
        for (int i = t; i < p.rank; i += DA_THREADS) a1_s[i] = p.proj[p.a1_off + i];
        __syncthreads();
    }
    for (int i = t; i < 4 * R; i += DA_THREADS) {
        float q = 0.f, k = 0.f, a = 0.f;
        if (i < p.dk) da_channel(p, p.proj, h * p.dk + i, gla ? da_dot_rank(a2_s + i * p.rank, a1_s, p.rank) : 0.f, q, k, a);
        q_s[i] = q;
        k_s[i] = k;
        a_s[i] = a;
    }
    __syncthreads();
    pdl_launch_dependents();
    const float4 *qv = reinterpret_cast<const float4*>(q_s + q4 * R), *kv = reinterpret_cast<const float4*>(k_s + q4 * R), *av = reinterpret_cast<const float4*>(a_s + q4 * R);
    float o0 = 0.f, o1 = 0.f;
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

// grid (H, ceil(dv / 64), segments), block 16 x 64 / C.  Thread (C columns, row sixteenth) holds R = dk_p / 16 rows of C columns as packed
// pairs of rows, so that the state update and the read-out are two-wide fp32 instructions and a row of q, k, a is read from shared memory
// once for C columns (with two columns those reads bounded the kernel).  Operands of DA_U tokens at a time come DA_AHEAD - 1 stages ahead by
// cp.async (a row part is padded so that eight neighbouring lanes' 16-byte reads sit on different banks); one block barrier per DA_U tokens,
// and no branch between the tokens of a full stage, so that the next token's operands are read under the present one's arithmetic.
#define DA_U 4
#define DA_AHEAD 3
#define DA_SLAB 64 /* columns per CTA */
__device__ __forceinline__ void da_cp16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void da_cp4(void* dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
typedef unsigned long long da_f2; // two fp32 values
__device__ __forceinline__ da_f2 da_pack(float x, float y) {
    da_f2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(x), "f"(y));
    return r;
}
__device__ __forceinline__ float2 da_unpack(da_f2 v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ da_f2 da_fma2(da_f2 a, da_f2 b, da_f2 c) {
    da_f2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ da_f2 da_mul2(da_f2 a, da_f2 b) {
    da_f2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
struct __align__(16) da_quad { da_f2 lo, hi; }; // four consecutive rows

// Segments (gridDim.z = P > 1; segment g is tokens g * seg .. of the chunk).  The state after a segment is diag(b) S_in + L, b the product
// of its decays and L what it makes of a zero state.  LOCAL (first launch): every segment leaves L and b in the workspace; segment 0 starts
// from the sequence's state, so its L is a true state.  Second launch: segment g makes its S_in from the L and b of those before it, then runs
// with read-outs; segment 0, the only one that touches the sequence's state, replaces it by the state after the last segment.
template <int R, int C, bool LOCAL>
__device__ __forceinline__ void da_scan_body(const lb_decay_params2& p) {
    constexpr int DA_SCAN_THREADS = 16 * DA_SLAB / C;
    constexpr int QS = R == 4 ? 4 : R + 4, VEC = 16 * QS, TOK = 3 * VEC + DA_SLAB; // floats: a row part, a vector, a token's operands
    constexpr int PV = 4 * R, PIECES = (LOCAL ? 2 : 3) * PV;                         // 16-byte pieces of a vector; of a token (no q for LOCAL)
    constexpr int NI = (DA_U * PIECES + DA_SCAN_THREADS - 1) / DA_SCAN_THREADS;
    extern __shared__ __align__(16) float da_sm[]; // [DA_AHEAD][DA_U][TOK]
    const int h = blockIdx.x, t = threadIdx.x, e = t & 15, cg = t >> 4, j = blockIdx.y * DA_SLAB + C * cg;
    const int g = blockIdx.z, P = gridDim.z, tok0 = g * p.seg, n_tok = min(p.seg, p.T - tok0), n_st = (n_tok + DA_U - 1) / DA_U;
    const int rows = min(R, p.dk - e * R), cols = min(C, p.dv - j); // what of this thread's tile exists
    const size_t head_off = ((size_t)h * p.dk + (size_t)e * R) * p.dv + j, all = (size_t)p.H * p.dk * p.dv; // this thread's corner of a state
    pdl_wait();
    // operands: a thread copies the same pieces of every stage, so only the source moves on.  A last stage reads past the chunk's tokens
    // (the buffers hold a whole number of stages); what it reads there is not used.
    const float* src[NI];
    int dst[NI];
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int idx = t + i * DA_SCAN_THREADS, u = idx / PIECES, c = idx - u * PIECES, which = c / PV + (LOCAL ? 1 : 0), pc = c % PV;
        src[i] = (which == 0 ? p.q : which == 1 ? p.k : p.a) + ((size_t)(tok0 + u) * p.H + h) * (16 * R) + pc * 4;
        dst[i] = u * TOK + which * VEC + (pc / (R / 4)) * QS + (pc % (R / 4)) * 4;
    }
    const float* vsrc = p.proj + (size_t)(tok0 + t / DA_SLAB) * p.ld + p.v_off + (size_t)h * p.dv + min(blockIdx.y * DA_SLAB + t % DA_SLAB, (unsigned)p.dv - 1u);
    const size_t step_qka = (size_t)DA_U * p.H * (16 * R), step_v = (size_t)DA_U * p.ld;
    int f_slot = 0;
    auto fetch = [&]() {
        float* d = da_sm + f_slot * (DA_U * TOK);
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            if ((i + 1) * DA_SCAN_THREADS <= DA_U * PIECES || t + i * DA_SCAN_THREADS < DA_U * PIECES) da_cp16(d + dst[i], src[i]);
            src[i] += step_qka;
        }
#pragma unroll
        for (int u = 0; u < DA_U; u += DA_SCAN_THREADS / DA_SLAB)
            da_cp4(d + (u + t / DA_SLAB) * TOK + 3 * VEC + t % DA_SLAB, vsrc + (size_t)u * p.ld);
        vsrc += step_v;
        if (++f_slot == DA_AHEAD) f_slot = 0;
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
#pragma unroll
    for (int st = 0; st < DA_AHEAD - 1; ++st) {
        if (st < n_st) fetch();
        else asm volatile("cp.async.commit_group;" ::: "memory");
    }
    // the tile as pairs of rows (2r, 2r + 1), column by column
    da_f2 s[C][R / 2];
    auto load = [&](const float* S) {
#pragma unroll
        for (int r = 0; r < R; r += 2)
#pragma unroll
            for (int c = 0; c < C; ++c)
                s[c][r / 2] = da_pack(c < cols && r < rows ? S[(size_t)r * p.dv + c] : 0.f, c < cols && r + 1 < rows ? S[(size_t)(r + 1) * p.dv + c] : 0.f);
    };
    auto store = [&](float* S) {
#pragma unroll
        for (int r = 0; r < R; r += 2)
#pragma unroll
            for (int c = 0; c < C; ++c) {
                const float2 x = da_unpack(s[c][r / 2]);
                if (c < cols && r < rows) S[(size_t)r * p.dv + c] = x.x;
                if (c < cols && r + 1 < rows) S[(size_t)(r + 1) * p.dv + c] = x.y;
            }
    };
    auto advance = [&](int seg) { // the state through a whole segment: S <- diag(b) S + L
        const float* L = p.seg_state + (size_t)seg * all + head_off;
        const float* b = p.seg_decay + ((size_t)seg * p.H + h) * (16 * R) + e * R;
#pragma unroll
        for (int r = 0; r < R; r += 2) {
            const da_f2 bb = da_pack(b[r], b[r + 1]);
#pragma unroll
            for (int c = 0; c < C; ++c)
                s[c][r / 2] = da_fma2(bb, s[c][r / 2], da_pack(c < cols && r < rows ? L[(size_t)r * p.dv + c] : 0.f, c < cols && r + 1 < rows ? L[(size_t)(r + 1) * p.dv + c] : 0.f));
        }
    };
    if (LOCAL ? g > 0 : false) {
#pragma unroll
        for (int c = 0; c < C; ++c)
#pragma unroll
            for (int r = 0; r < R / 2; ++r) s[c][r] = 0ull;
    } else if (LOCAL || g == 0) {
        load(p.state + head_off);
    } else {
        load(p.seg_state + head_off);
        for (int q = 1; q < g; ++q) advance(q);
    }
    da_f2 dec[R / 2]; // LOCAL: product of the segment's decays
#pragma unroll
    for (int r = 0; r < R / 2; ++r) dec[r] = da_pack(1.f, 1.f);

    auto step = [&](const float* tk, int tok) { // one token: state update, read-out
        float v[C];
#pragma unroll
        for (int c = 0; c < C; c += 4) {
            const float4 x = *reinterpret_cast<const float4*>(tk + 3 * VEC + C * cg + c);
            v[c] = x.x; v[c + 1] = x.y; v[c + 2] = x.z; v[c + 3] = x.w;
        }
        const da_quad *qv = reinterpret_cast<const da_quad*>(tk + e * QS), *kv = reinterpret_cast<const da_quad*>(tk + VEC + e * QS),
                      *av = reinterpret_cast<const da_quad*>(tk + 2 * VEC + e * QS);
        da_f2 acc[C];
#pragma unroll
        for (int c = 0; c < C; ++c) acc[c] = 0ull;
#pragma unroll
        for (int i = 0; i < R / 4; ++i) {
            const da_quad k = kv[i], a = av[i];
            da_quad q;
            if (!LOCAL) q = qv[i];
#pragma unroll
            for (int c = 0; c < C; ++c) {
                const da_f2 vv = da_pack(v[c], v[c]);
                s[c][2 * i] = da_fma2(a.lo, s[c][2 * i], da_mul2(k.lo, vv));
                s[c][2 * i + 1] = da_fma2(a.hi, s[c][2 * i + 1], da_mul2(k.hi, vv));
                if (!LOCAL) acc[c] = da_fma2(s[c][2 * i + 1], q.hi, da_fma2(s[c][2 * i], q.lo, acc[c]));
            }
            if (LOCAL) {
                dec[2 * i] = da_mul2(dec[2 * i], a.lo);
                dec[2 * i + 1] = da_mul2(dec[2 * i + 1], a.hi);
            }
        }
        if (LOCAL) return;
        float o[C];
#pragma unroll
        for (int c = 0; c < C; ++c) {
            const float2 x = da_unpack(acc[c]);
            o[c] = x.x + x.y;
        }
        // sums over the 16 row parts: each of the first exchanges halves what a lane still holds, the others add two lanes
        int bit = 8;
#pragma unroll
        for (int half = C / 2; half >= 1; half >>= 1, bit >>= 1) {
            const bool up = (e & bit) != 0;
#pragma unroll
            for (int i = 0; i < half; ++i) {
                const float give = up ? o[i] : o[i + half], keep = up ? o[i + half] : o[i];
                o[i] = keep + __shfl_xor_sync(0xffffffffu, give, bit);
            }
        }
#pragma unroll
        for (; bit >= 1; bit >>= 1) o[0] += __shfl_xor_sync(0xffffffffu, o[0], bit);
        const int col = e / (16 / C);
        if (e % (16 / C) == 0 && col < cols) p.o[((size_t)(tok0 + tok) * p.H + h) * p.dv + j + col] = o[0];
    };
    int slot = 0;
    for (int st = 0; st < n_st; ++st) {
        asm volatile("cp.async.wait_group %0;" ::"n"(DA_AHEAD - 2) : "memory");
        __syncthreads(); // everybody's pieces have landed, and everybody is done with the stage the next fetch fills
        if (st + DA_AHEAD - 1 < n_st) fetch();
        else asm volatile("cp.async.commit_group;" ::: "memory");
        const float* base = da_sm + slot * (DA_U * TOK);
        if (++slot == DA_AHEAD) slot = 0;
        if ((st + 1) * DA_U <= n_tok) {
#pragma unroll
            for (int u = 0; u < DA_U; ++u) step(base + u * TOK, st * DA_U + u);
        } else { // the segment ends inside this stage: tokens past it leave the state alone
            for (int u = 0; st * DA_U + u < n_tok; ++u) step(base + u * TOK, st * DA_U + u);
        }
    }
    pdl_launch_dependents();
    if (LOCAL) {
        store(p.seg_state + (size_t)g * all + head_off);
        if (blockIdx.y == 0 && t < 16) {
            float* b = p.seg_decay + ((size_t)g * p.H + h) * (16 * R) + e * R;
#pragma unroll
            for (int r = 0; r < R / 2; ++r) {
                const float2 x = da_unpack(dec[r]);
                b[2 * r] = x.x;
                b[2 * r + 1] = x.y;
            }
        }
    } else if (P == 1) {
        store(p.state + head_off);
    } else if (g == 0) {
        load(p.seg_state + head_off);
        for (int q = 1; q < P; ++q) advance(q);
        store(p.state + head_off);
    }
}
#define DA_SCAN_KERNELS(dk, R, C)                                                                                                                                          \
    extern "C" __global__ void __launch_bounds__(16 * DA_SLAB / C) da_scan_##dk(const __grid_constant__ lb_decay_params2 p) { da_scan_body<R, C, false>(p); } \
    extern "C" __global__ void __launch_bounds__(16 * DA_SLAB / C) da_local_##dk(const __grid_constant__ lb_decay_params2 p) { da_scan_body<R, C, true>(p); }
DA_SCAN_KERNELS(64, 4, 8)
DA_SCAN_KERNELS(128, 8, 8)
DA_SCAN_KERNELS(256, 16, 4)

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
