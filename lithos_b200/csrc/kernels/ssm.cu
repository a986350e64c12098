// State-space recurrence with a scalar decay per head:  S <- exp(-exp(A_log) dt) S + dt B x^T,  y = S^T C + D x,  where x, B and C have passed a
// causal convolution per channel and silu, and dt = softplus(projection + bias).  B and C belong to a group of heads.  States, step sizes,
// decays and read-outs are fp32.
// A column of a head's state needs only that column of x, so a CTA owns LB_SSM_COLS columns of one head.
//   ssm_step_*     one token (decode): convolution, state read and written once, read-out
//   ssm_conv       a prompt chunk's convolved channels and step sizes
//   ssm_chunk_*    a prompt chunk on the tensor cores, block by block of LB_SSM_SEG tokens, the state on chip between blocks; where the heads
//                  are few, in segments side by side: ssm_local_* carries each from a zero state, ssm_chunk_* starts each from its true state
//   ssm_scan_f32_* the same token by token in fp32
//   ssm_finish     gate, norm in parts, and the convolution's last inputs into the ring
#include "mma_sync.cuh"
#include "params.h"

__device__ __forceinline__ float sm_silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float sm_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// sum over the earlier taps of channel ch at position pos (bias included): values of earlier positions from the ring, nothing before the start
__device__ __forceinline__ float sm_conv_past(const lb_ssm_params& p, int ch, int pos) {
    float s = bf16_bits_to_f32(p.conv_b[ch]);
    for (int k = p.taps - 1; k >= 1; --k)
        if (pos >= k) s = fmaf(bf16_bits_to_f32(p.conv_w[(size_t)ch * p.taps + p.taps - 1 - k]), p.ring[(size_t)((pos - k) % p.taps) * p.channels + ch], s);
    return s;
}

// grid (H, ceil(V / 32)), block 128: thread (column, quarter of the state's rows).  The state and the ring (written a whole step ago) and the
// constants are under way before the wait for the projections.
template <int R>
__device__ __forceinline__ void ssm_step_body(const lb_ssm_params& p) {
    __shared__ __align__(16) float b_s[4 * R], c_s[4 * R];
    __shared__ float x_s[LB_SSM_COLS];
    const int h = blockIdx.x, t = threadIdx.x, q4 = t & 3, j = blockIdx.y * LB_SSM_COLS + (t >> 2);
    const int pos = p.pos_ptr[0], inner = p.H * p.V, hg = p.H / p.G, g = h / hg;
    const bool live = j < p.V;
    float* S = p.state + ((size_t)h * p.N + (size_t)q4 * R) * p.V + j;
    const int rows = min(R, p.N - q4 * R);
    float s[R];
#pragma unroll
    for (int r = 0; r < R; ++r) s[r] = live && r < rows ? S[(size_t)r * p.V] : 0.f;
    // channels of this CTA: N of B, N of C, 32 of x; a thread has up to five of them
    constexpr int NI = (8 * R + LB_SSM_COLS + 127) / 128;
    const int n_ch = 2 * p.N + LB_SSM_COLS;
    int chan[NI];
    float past[NI];
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int e = t + 128 * i, c = e - 2 * p.N;
        chan[i] = -1;
        past[i] = 0.f;
        if (e < p.N) chan[i] = inner + g * p.N + e;
        else if (e < 2 * p.N) chan[i] = inner + p.G * p.N + g * p.N + (e - p.N);
        else if (e < n_ch && (int)blockIdx.y * LB_SSM_COLS + c < p.V) chan[i] = h * p.V + blockIdx.y * LB_SSM_COLS + c;
        if (chan[i] >= 0) past[i] = sm_conv_past(p, chan[i], pos);
    }
    const float a_neg = -expf(bf16_bits_to_f32(p.a_log[h])), bias = bf16_bits_to_f32(p.dt_bias[h]), dskip = bf16_bits_to_f32(p.d[h]);
    for (int i = p.N + t; i < 4 * R; i += 128) b_s[i] = c_s[i] = 0.f;
    pdl_wait();
    const float dt = sm_softplus(p.proj[2 * inner + 2 * p.G * p.N + h] + bias), decay = expf(a_neg * dt);
    float* slot = p.ring + (size_t)(pos % p.taps) * p.channels;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        if (chan[i] < 0) continue;
        const int e = t + 128 * i, ch = chan[i];
        const float cur = p.proj[inner + ch], v = sm_silu(fmaf(bf16_bits_to_f32(p.conv_w[(size_t)ch * p.taps + p.taps - 1]), cur, past[i]));
        if (e < p.N) b_s[e] = v;
        else if (e < 2 * p.N) c_s[e - p.N] = v;
        else x_s[e - 2 * p.N] = v;
        if (e >= 2 * p.N || (blockIdx.y == 0 && h == g * hg)) slot[ch] = cur; // nobody reads this slot during this step
    }
    __syncthreads();
    pdl_launch_dependents();
    const float x = live ? x_s[t >> 2] : 0.f, dx = dt * x;
    float o0 = 0.f, o1 = 0.f;
    const float4 *bv = reinterpret_cast<const float4*>(b_s + q4 * R), *cv = reinterpret_cast<const float4*>(c_s + q4 * R);
#pragma unroll
    for (int c = 0; c < R / 4; ++c) {
        const float4 b = bv[c], k = cv[c];
        s[4 * c] = fmaf(decay, s[4 * c], b.x * dx);
        s[4 * c + 1] = fmaf(decay, s[4 * c + 1], b.y * dx);
        s[4 * c + 2] = fmaf(decay, s[4 * c + 2], b.z * dx);
        s[4 * c + 3] = fmaf(decay, s[4 * c + 3], b.w * dx);
        o0 = fmaf(s[4 * c], k.x, o0);
        o1 = fmaf(s[4 * c + 1], k.y, o1);
        o0 = fmaf(s[4 * c + 2], k.z, o0);
        o1 = fmaf(s[4 * c + 3], k.w, o1);
    }
#pragma unroll
    for (int r = 0; r < R; ++r)
        if (live && r < rows) S[(size_t)r * p.V] = s[r];
    float o = o0 + o1;
    o += __shfl_xor_sync(0xffffffffu, o, 1);
    o += __shfl_xor_sync(0xffffffffu, o, 2);
    if (live && q4 == 0) p.y[(size_t)h * p.V + j] = fmaf(dskip, x, o);
}
extern "C" __global__ void __launch_bounds__(128) ssm_step_64(const __grid_constant__ lb_ssm_params p) { ssm_step_body<16>(p); }
extern "C" __global__ void __launch_bounds__(128) ssm_step_128(const __grid_constant__ lb_ssm_params p) { ssm_step_body<32>(p); }
extern "C" __global__ void __launch_bounds__(128) ssm_step_256(const __grid_constant__ lb_ssm_params p) { ssm_step_body<64>(p); }

// grid (ceil((ld_xbc + H) / 256), ceil(T / 16)), block 256: a thread makes one (padded) channel, or one head's step sizes, of LB_SSM_CONV_TOKENS tokens
extern "C" __global__ void __launch_bounds__(256) ssm_conv(const __grid_constant__ lb_ssm_params p) {
    const int i = blockIdx.x * 256 + threadIdx.x, t0 = blockIdx.y * LB_SSM_CONV_TOKENS, nt = min(LB_SSM_CONV_TOKENS, p.T - t0), inner = p.H * p.V;
    const int nx = p.H * p.V_p, nb = p.G * p.N_p;
    pdl_wait();
    if (i < p.ld_xbc) {
        int ch = -1;
        if (i < nx) {
            const int h = i / p.V_p, j = i - h * p.V_p;
            if (j < p.V) ch = h * p.V + j;
        } else {
            const int k = i - nx, c = k >= nb, e = k - c * nb, g = e / p.N_p, n = e - g * p.N_p;
            if (n < p.N) ch = inner + c * p.G * p.N + g * p.N + n;
        }
        float w[LB_SSM_MAX_TAPS], past[LB_SSM_MAX_TAPS]; // lag k: weight, value k tokens ago
        float bias = 0.f;
        if (ch >= 0) {
            bias = bf16_bits_to_f32(p.conv_b[ch]);
#pragma unroll
            for (int k = 0; k < LB_SSM_MAX_TAPS; ++k) {
                w[k] = past[k] = 0.f;
                if (k >= p.taps) continue;
                w[k] = bf16_bits_to_f32(p.conv_w[(size_t)ch * p.taps + p.taps - 1 - k]);
                const int s = t0 - k, pos = p.pos0 + s;
                if (k > 0 && pos >= 0) past[k] = s >= 0 ? p.proj[(size_t)s * p.ld + inner + ch] : p.ring[(size_t)(pos % p.taps) * p.channels + ch];
            }
        }
        float cur[LB_SSM_CONV_TOKENS];
#pragma unroll
        for (int u = 0; u < LB_SSM_CONV_TOKENS; ++u) cur[u] = ch >= 0 && u < nt ? __ldcs(p.proj + (size_t)(t0 + u) * p.ld + inner + ch) : 0.f;
#pragma unroll
        for (int u = 0; u < LB_SSM_CONV_TOKENS; ++u) {
            if (u >= nt) break;
            float v = 0.f;
            if (ch >= 0) {
                past[0] = cur[u];
                float s = bias;
#pragma unroll
                for (int k = LB_SSM_MAX_TAPS - 1; k >= 0; --k) s = fmaf(w[k], past[k], s);
                v = sm_silu(s);
#pragma unroll
                for (int k = LB_SSM_MAX_TAPS - 1; k >= 1; --k) past[k] = past[k - 1];
            }
            const size_t o = (size_t)(t0 + u) * p.ld_xbc + i;
            if (p.f32) reinterpret_cast<float*>(p.xbc)[o] = v;
            else reinterpret_cast<__nv_bfloat16*>(p.xbc)[o] = __float2bfloat16_rn(v);
        }
    } else if (i - p.ld_xbc < p.H) {
        const int h = i - p.ld_xbc;
        const float bias = bf16_bits_to_f32(p.dt_bias[h]);
        for (int u = 0; u < nt; ++u) p.dt[(size_t)(t0 + u) * p.H + h] = sm_softplus(p.proj[(size_t)(t0 + u) * p.ld + 2 * inner + 2 * p.G * p.N + h] + bias);
    }
    pdl_launch_dependents();
}

// grid (H, ceil(V / 32), segments), block 128 (4 warps).  With c_i the sum of a = -exp(A_log) dt over the block's tokens up to i, a block of tokens does
//   y_i = exp(c_i) S^T C_i + sum_(j <= i) exp(c_i - c_j) dt_j (C_i . B_j) x_j + D x_i
//   S  <- exp(c_end) S + sum_j B_j (exp(c_end - c_j) dt_j x_j)^T
// as products mma.sync m16n8k16: B, C and x are bf16 (the convolution's activations); the fp32 factors -- the state, the weights of (i, j), the
// scaled x -- enter as three bf16 terms, which carry all their 24 bits; sums are fp32.  Warp w has tokens 16 w .. 16 w + 15 of the block as
// rows of y, and the state rows of the tiles w, w + 4, ... (MT of them) in registers.
// dynamic shared memory: B, C [64][N_p + 8], x [64][40], S terms [3][N_p][40], scaled x terms [3][64][40] (in C's place where they fit, so that
// three CTAs share an SM), all bf16; c, dt [64] fp32
// Segments (gridDim.z = P > 1; segment g is tokens g * seg .. of the chunk): LOCAL (first launch, P - 1 segments) leaves what each segment makes of
// a zero state (segment 0: of the sequence's state) and its summed log decay, and keeps the sequence's state in the last place; the second
// launch makes a segment's start from those before it, and the last segment leaves the sequence's state.
#define SC_XST 80 /* bytes of a row of 32 columns and 16 bytes of padding */
template <int MT, bool LOCAL>
__device__ __forceinline__ void ssm_chunk_body(const lb_ssm_params& p) {
    extern __shared__ __align__(16) unsigned char sc_sm[];
    const int t = threadIdx.x, lane = t & 31, warp = t >> 5, fg = lane >> 2, ft = lane & 3;
    const int h = blockIdx.x, col0 = blockIdx.y * LB_SSM_COLS, g = h / (p.H / p.G);
    const int bst = 2 * p.N_p + 16, n16 = p.N_p / 8, nk = p.N_p / 16;
    unsigned char *b_s = sc_sm, *c_s = b_s + LB_SSM_SEG * bst, *x_s = c_s + LB_SSM_SEG * bst, *s_s = x_s + LB_SSM_SEG * SC_XST,
                  *end_s = s_s + 3 * p.N_p * SC_XST;
    const bool shared_w = bst >= 3 * SC_XST;
    unsigned char* w_s = shared_w ? c_s : end_s;
    float* cum = reinterpret_cast<float*>(end_s + (shared_w ? 0 : 3 * LB_SSM_SEG * SC_XST));
    float* dts = cum + LB_SSM_SEG;
    const uint32_t s_term = p.N_p * SC_XST, w_term = LB_SSM_SEG * SC_XST;
    const float a_neg = -expf(bf16_bits_to_f32(p.a_log[h])), dskip = bf16_bits_to_f32(p.d[h]);
    const int seg = blockIdx.z, P = LOCAL ? gridDim.z + 1 : gridDim.z, tok_lo = seg * p.seg, tok_hi = min(p.T, tok_lo + p.seg);
    const int n_blk = (tok_hi - tok_lo + LB_SSM_SEG - 1) / LB_SSM_SEG;
    pdl_wait();
    const uint16_t* xbc = reinterpret_cast<const uint16_t*>(p.xbc);
    const uint16_t *gx = xbc + (size_t)h * p.V_p + col0, *gb = xbc + (size_t)p.H * p.V_p + (size_t)g * p.N_p, *gc = gb + (size_t)p.G * p.N_p;
    // tokens past the segment repeat its last one (finite values); their step size is 0 and they are not stored
    auto load = [&](int blk) {
        for (int r = warp; r < LB_SSM_SEG; r += 4) {
            const size_t row = (size_t)min(tok_lo + blk * LB_SSM_SEG + r, tok_hi - 1) * p.ld_xbc;
            for (int c = lane; c < n16; c += 32) {
                ms_cp16(smem_u32(b_s + r * bst + c * 16), gb + row + c * 8);
                if (!LOCAL) ms_cp16(smem_u32(c_s + r * bst + c * 16), gc + row + c * 8);
            }
            if (lane < 4) ms_cp16(smem_u32(x_s + r * SC_XST + lane * 16), gx + row + lane * 8);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load(0);

    // the state: tile mt of this warp is rows 16 (warp + 4 mt) + fg (+ 8), columns 8 nt + 2 ft (+ 1)
    float st[MT][4][4];
    const size_t corner = (size_t)h * p.N * p.V + col0, all = (size_t)p.H * p.N * p.V;
    auto each = [&](auto f) { // f(value, offset from the head's corner) of what exists of the state
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
            for (int nt = 0; nt < 4; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int n = 16 * (warp + 4 * mt) + fg + 8 * (e >> 1), c = 8 * nt + 2 * ft + (e & 1);
                    if (n < p.N && col0 + c < p.V) f(st[mt][nt][e], (size_t)n * p.V + c);
                }
    };
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int nt = 0; nt < 4; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) st[mt][nt][e] = 0.f;
    float* first = P > 1 ? p.seg_state + (size_t)(P - 1) * all + corner : nullptr; // the sequence's state, kept
    if (LOCAL ? seg == 0 : P == 1) {
        each([&](float& v, size_t o) { v = p.state[corner + o]; });
        if (LOCAL) each([&](float& v, size_t o) { first[o] = v; });
    } else if (!LOCAL && seg == 0) {
        each([&](float& v, size_t o) { v = first[o]; });
    } else if (!LOCAL) {
        each([&](float& v, size_t o) { v = p.seg_state[corner + o]; });
        for (int q = 1; q < seg; ++q) {
            const float d = expf(p.seg_decay[(size_t)q * p.H + h]);
            each([&](float& v, size_t o) { v = fmaf(d, v, p.seg_state[(size_t)q * all + corner + o]); });
        }
    }
    float log_decay = 0.f; // LOCAL: of the segment so far
    auto put_state = [&]() {
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
            const int tile = warp + 4 * mt;
            if (tile >= nk) continue;
#pragma unroll
            for (int nt = 0; nt < 4; ++nt)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    uint32_t a, b, c;
                    ms_split3(st[mt][nt][2 * e], st[mt][nt][2 * e + 1], a, b, c);
                    unsigned char* d = s_s + (16 * tile + fg + 8 * e) * SC_XST + (8 * nt + 2 * ft) * 2;
                    *reinterpret_cast<uint32_t*>(d) = a;
                    *reinterpret_cast<uint32_t*>(d + s_term) = b;
                    *reinterpret_cast<uint32_t*>(d + 2 * s_term) = c;
                }
        }
    };
    if (!LOCAL) put_state();
    const uint32_t a_row = (warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * bst + (lane >> 4) * 16; // A operand: rows of C
    const uint32_t k_row = ((lane & 7) + ((lane >> 4) << 3)) * bst + ((lane >> 3) & 1) * 16;          // B operand: rows of B as columns
    const uint32_t t_row = ((lane & 7) + ((lane >> 3) & 1) * 8) * SC_XST + (lane >> 4) * 16;          // B operand: rows are k (transposing load)
    const uint32_t ta_row = ((lane & 7) + ((lane >> 4) << 3)) * bst + ((lane >> 3) & 1) * 16;         // A operand: rows of B are k (transposing load)
    const uint32_t ub = smem_u32(b_s), uc = smem_u32(c_s), ux = smem_u32(x_s), us = smem_u32(s_s), uw = smem_u32(w_s);

    for (int blk = 0; blk < n_blk; ++blk) {
        const int tok0 = tok_lo + blk * LB_SSM_SEG;
        if (warp == 0) { // step sizes and the running sum of log decays: lane has tokens 2 lane, 2 lane + 1
            const int i0 = tok0 + 2 * lane;
            const float d0 = i0 < tok_hi ? p.dt[(size_t)i0 * p.H + h] : 0.f, d1 = i0 + 1 < tok_hi ? p.dt[(size_t)(i0 + 1) * p.H + h] : 0.f;
            const float a0 = a_neg * d0, a1 = a_neg * d1;
            float s = a0 + a1;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float v = __shfl_up_sync(0xffffffffu, s, o);
                if (lane >= o) s += v;
            }
            cum[2 * lane] = s - a1;
            cum[2 * lane + 1] = s;
            dts[2 * lane] = d0;
            dts[2 * lane + 1] = d1;
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        const float c_end = cum[LB_SSM_SEG - 1];
        if (!LOCAL) { // C . B and C . S of the warp's 16 tokens
        float sc[8][4], y[4][4];
#pragma unroll
        for (int j = 0; j < 8; ++j) sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.f;
#pragma unroll
        for (int j = 0; j < 4; ++j) y[j][0] = y[j][1] = y[j][2] = y[j][3] = 0.f;
#pragma unroll 2
        for (int k = 0; k < nk; ++k) {
            uint32_t a0, a1, a2, a3;
            ms_ldsm(uc + a_row + k * 32, a0, a1, a2, a3);
#pragma unroll
            for (int jj = 0; jj < 4; ++jj) {
                if (jj > warp) continue; // later tokens
                uint32_t b0, b1, b2, b3;
                ms_ldsm(ub + k_row + jj * 16 * bst + k * 32, b0, b1, b2, b3);
                ms_mma(sc[2 * jj], a0, a1, a2, a3, b0, b1);
                ms_mma(sc[2 * jj + 1], a0, a1, a2, a3, b2, b3);
            }
#pragma unroll
            for (int term = 2; term >= 0; --term)
#pragma unroll
                for (int nn = 0; nn < 2; ++nn) {
                    uint32_t v0, v1, v2, v3;
                    ms_ldsm_t(us + term * s_term + t_row + k * 16 * SC_XST + nn * 32, v0, v1, v2, v3);
                    ms_mma(y[2 * nn], a0, a1, a2, a3, v0, v1);
                    ms_mma(y[2 * nn + 1], a0, a1, a2, a3, v2, v3);
                }
        }
        const int i0 = warp * 16 + fg;
        const float ci[2] = {cum[i0], cum[i0 + 8]}, ei[2] = {expf(ci[0]), expf(ci[1])};
#pragma unroll
        for (int j = 0; j < 4; ++j) { y[j][0] *= ei[0]; y[j][1] *= ei[0]; y[j][2] *= ei[1]; y[j][3] *= ei[1]; }
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) { // 16 earlier tokens at a time
            if (kk > warp) continue;
            uint32_t m[3][4];
#pragma unroll
            for (int q = 0; q < 4; ++q) { // fragment registers: (rows fg, fg + 8) x (columns 2 ft, 2 ft + 8)
                const int r = q & 1, nt = 2 * kk + (q >> 1), j = 8 * nt + 2 * ft;
                const float2 cj = *reinterpret_cast<const float2*>(cum + j), dj = *reinterpret_cast<const float2*>(dts + j);
                const int i = i0 + 8 * r;
                const float e0 = j <= i ? expf(ci[r] - cj.x) * dj.x : 0.f, e1 = j + 1 <= i ? expf(ci[r] - cj.y) * dj.y : 0.f;
                ms_split3(sc[nt][2 * r] * e0, sc[nt][2 * r + 1] * e1, m[0][q], m[1][q], m[2][q]);
            }
#pragma unroll
            for (int nn = 0; nn < 2; ++nn) {
                uint32_t v0, v1, v2, v3;
                ms_ldsm_t(ux + t_row + kk * 16 * SC_XST + nn * 32, v0, v1, v2, v3);
#pragma unroll
                for (int term = 2; term >= 0; --term) {
                    ms_mma(y[2 * nn], m[term][0], m[term][1], m[term][2], m[term][3], v0, v1);
                    ms_mma(y[2 * nn + 1], m[term][0], m[term][1], m[term][2], m[term][3], v2, v3);
                }
            }
        }
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int tok = tok0 + i0 + 8 * r;
            if (tok >= tok_hi) continue;
            float* dst = p.y + ((size_t)tok * p.H + h) * p.V + col0;
#pragma unroll
            for (int nt = 0; nt < 4; ++nt) {
                const int c = 8 * nt + 2 * ft;
                const uint32_t u = *reinterpret_cast<const uint32_t*>(x_s + (i0 + 8 * r) * SC_XST + c * 2);
                if (col0 + c < p.V) dst[c] = fmaf(dskip, __uint_as_float(u << 16), y[nt][2 * r]);
                if (col0 + c + 1 < p.V) dst[c + 1] = fmaf(dskip, __uint_as_float(u & 0xffff0000u), y[nt][2 * r + 1]);
            }
        }
        }
        if (!LOCAL) __syncthreads(); // C and the old state's terms have been read
        log_decay += c_end;
        // scaled x
        for (int i = t; i < LB_SSM_SEG * 16; i += 128) {
            const int r = i >> 4, c = i & 15;
            const float w = dts[r] * expf(c_end - cum[r]);
            const uint32_t u = *reinterpret_cast<const uint32_t*>(x_s + r * SC_XST + c * 4);
            uint32_t a, b, d;
            ms_split3(w * __uint_as_float(u << 16), w * __uint_as_float(u & 0xffff0000u), a, b, d);
            unsigned char* dst = w_s + r * SC_XST + c * 4;
            *reinterpret_cast<uint32_t*>(dst) = a;
            *reinterpret_cast<uint32_t*>(dst + w_term) = b;
            *reinterpret_cast<uint32_t*>(dst + 2 * w_term) = d;
        }
        __syncthreads();
        const float e_end = expf(c_end);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
            const int tile = warp + 4 * mt;
            if (tile >= nk) continue;
#pragma unroll
            for (int nt = 0; nt < 4; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) st[mt][nt][e] *= e_end;
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) {
                uint32_t a0, a1, a2, a3;
                ms_ldsm_t(ub + ta_row + kk * 16 * bst + tile * 32, a0, a1, a2, a3);
#pragma unroll
                for (int term = 2; term >= 0; --term)
#pragma unroll
                    for (int nn = 0; nn < 2; ++nn) {
                        uint32_t v0, v1, v2, v3;
                        ms_ldsm_t(uw + term * w_term + t_row + kk * 16 * SC_XST + nn * 32, v0, v1, v2, v3);
                        ms_mma(st[mt][2 * nn], a0, a1, a2, a3, v0, v1);
                        ms_mma(st[mt][2 * nn + 1], a0, a1, a2, a3, v2, v3);
                    }
            }
        }
        if (blk + 1 < n_blk) {
            if (!LOCAL) put_state();
            __syncthreads(); // everybody is done with B, x, scaled x, c and dt
            load(blk + 1);
        }
    }
    pdl_launch_dependents();
    if (LOCAL) {
        each([&](float& v, size_t o) { p.seg_state[(size_t)seg * all + corner + o] = v; });
        if (blockIdx.y == 0 && t == 0) p.seg_decay[(size_t)seg * p.H + h] = log_decay;
    } else if (seg == P - 1) {
        each([&](float& v, size_t o) { p.state[corner + o] = v; });
    }
}
#define SC_KERNELS(n, MT, BLOCKS)                                                                                                                            \
    extern "C" __global__ void __launch_bounds__(128, BLOCKS) ssm_chunk_##n(const __grid_constant__ lb_ssm_params p) { ssm_chunk_body<MT, false>(p); } \
    extern "C" __global__ void __launch_bounds__(128, BLOCKS) ssm_local_##n(const __grid_constant__ lb_ssm_params p) { ssm_chunk_body<MT, true>(p); }
SC_KERNELS(64, 1, 3)
SC_KERNELS(128, 2, 3)
SC_KERNELS(256, 4, 1)

// fp32: grid (H, ceil(V / 32)), block 128, threads as in ssm_step; the operands of SF_TOK tokens at a time in shared memory
#define SF_TOK 8
template <int R>
__device__ __forceinline__ void ssm_scan_f32_body(const lb_ssm_params& p) {
    __shared__ __align__(16) float b_s[SF_TOK][4 * R], c_s[SF_TOK][4 * R], x_s[SF_TOK][LB_SSM_COLS], dt_s[SF_TOK];
    const int h = blockIdx.x, t = threadIdx.x, q4 = t & 3, j = blockIdx.y * LB_SSM_COLS + (t >> 2), g = h / (p.H / p.G);
    const bool live = j < p.V;
    float* S = p.state + ((size_t)h * p.N + (size_t)q4 * R) * p.V + j;
    const int rows = min(R, p.N - q4 * R);
    const float a_neg = -expf(bf16_bits_to_f32(p.a_log[h])), dskip = bf16_bits_to_f32(p.d[h]);
    pdl_wait();
    float s[R];
#pragma unroll
    for (int r = 0; r < R; ++r) s[r] = live && r < rows ? S[(size_t)r * p.V] : 0.f;
    const float* xbc = reinterpret_cast<const float*>(p.xbc);
    for (int t0 = 0; t0 < p.T; t0 += SF_TOK) {
        const int nt = min(SF_TOK, p.T - t0);
        __syncthreads();
        for (int u = 0; u < nt; ++u) {
            const float* row = xbc + (size_t)(t0 + u) * p.ld_xbc;
            for (int i = t; i < 4 * R; i += 128) {
                b_s[u][i] = i < p.N ? row[p.H * p.V_p + g * p.N_p + i] : 0.f;
                c_s[u][i] = i < p.N ? row[p.H * p.V_p + p.G * p.N_p + g * p.N_p + i] : 0.f;
            }
            if (t < LB_SSM_COLS) x_s[u][t] = row[(size_t)h * p.V_p + blockIdx.y * LB_SSM_COLS + t];
            if (t == 0) dt_s[u] = p.dt[(size_t)(t0 + u) * p.H + h];
        }
        __syncthreads();
        for (int u = 0; u < nt; ++u) {
            const float x = x_s[u][t >> 2], dx = dt_s[u] * x, decay = expf(a_neg * dt_s[u]);
            float o = 0.f;
#pragma unroll
            for (int r = 0; r < R; ++r) {
                s[r] = fmaf(decay, s[r], b_s[u][q4 * R + r] * dx);
                o = fmaf(s[r], c_s[u][q4 * R + r], o);
            }
            o += __shfl_xor_sync(0xffffffffu, o, 1);
            o += __shfl_xor_sync(0xffffffffu, o, 2);
            if (live && q4 == 0) p.y[((size_t)(t0 + u) * p.H + h) * p.V + j] = fmaf(dskip, x, o);
        }
    }
    pdl_launch_dependents();
#pragma unroll
    for (int r = 0; r < R; ++r)
        if (live && r < rows) S[(size_t)r * p.V] = s[r];
}
extern "C" __global__ void __launch_bounds__(128) ssm_scan_f32_64(const __grid_constant__ lb_ssm_params p) { ssm_scan_f32_body<16>(p); }
extern "C" __global__ void __launch_bounds__(128) ssm_scan_f32_128(const __grid_constant__ lb_ssm_params p) { ssm_scan_f32_body<32>(p); }
extern "C" __global__ void __launch_bounds__(128) ssm_scan_f32_256(const __grid_constant__ lb_ssm_params p) { ssm_scan_f32_body<64>(p); }

// cat[t] = norm in parts of (y[t] * silu(z[t])) * norm_w; the projections of the chunk's last `taps` tokens go to the ring.
// grid (T, norm_groups), block 128; dynamic shared memory: a part's values, fp32
extern "C" __global__ void __launch_bounds__(128) ssm_finish(const __grid_constant__ lb_ssm_params p) {
    extern __shared__ float sf_v[];
    __shared__ float red[40];
    const int s = blockIdx.x, n = p.H * p.V / p.norm_groups, o = blockIdx.y * n, t = threadIdx.x;
    pdl_wait();
    const float *y = p.y + (size_t)s * p.H * p.V + o, *z = p.proj + (size_t)s * p.ld + o;
    float ss = 0.f;
    for (int i = t; i < n; i += 128) {
        const float v = y[i] * sm_silu(z[i]);
        sf_v[i] = v;
        ss += v * v;
    }
    const float r = 1.0f / sqrtf(block_sum(ss, red) / (float)n + p.eps);
    for (int i = t; i < n; i += 128) {
        const float v = sf_v[i] * r * bf16_bits_to_f32(p.norm_w[o + i]);
        const size_t d = (size_t)s * p.cat_ld + o + i;
        if (p.f32) reinterpret_cast<float*>(p.cat)[d] = v;
        else reinterpret_cast<__nv_bfloat16*>(p.cat)[d] = __float2bfloat16_rn(v);
    }
    if (s >= p.T - p.taps)
        for (int i = blockIdx.y * 128 + t; i < p.channels; i += 128 * gridDim.y)
            p.ring[(size_t)((p.pos0 + s) % p.taps) * p.channels + i] = p.proj[(size_t)s * p.ld + p.H * p.V + i];
    pdl_launch_dependents();
}
