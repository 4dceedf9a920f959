// The gated delta rule with a decay per head and key channel, or one per head, over per-sequence state.
//
// Per head, with the state S [d, dv] float32 (zero when a sequence starts), for every token in order:
//     S <- diag(g_t) S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t
// so the read-out sees the token's own write.  Before that, per token (delta_prep_kernel):
//     q, k, v  = silu(conv(projection))     a causal convolution over time per channel, `taps` wide, the last
//                                           tap the token's own, zeros before the sequence's start
//     q, k     = x / sqrt(sum(x^2) + 1e-6) per head;  q also times q_scale
//     beta     = sigmoid(b)                 one per head
//     g        = exp(-exp(A_log_h) * softplus(a + dt_bias))      one per head and key channel, or one per head
// Query/key head of value head h: h / (heads / kv_heads).  The last taps - 1 rows of the raw q, k, v projections
// are per-sequence state as well ([taps - 1, channels] behind S in a slot's row), renewed by conv_state_kernel
// after the preparation has read them.  Everything here is float32 in both modes of the engine.
//
// delta_scan_kernel: the columns of S never meet, so a block owns (sequence, head, a group of columns); a column's
// d rows are spread over L lanes (L the smallest power of two that leaves a thread at most 32 rows; heads of up to
// 512 key channels) and live in registers for the whole step.  The step's tokens are staged through shared memory in tiles.  The two dot
// products of a token are added over the L lanes by a fixed tree of shuffles, and a token's arithmetic does not
// depend on where the step's cut falls, so prompts, portions and single tokens give the same bits.
//
// delta_chunk_scan_kernel: the same with one decay per head, eight tokens at a time, for steps where that order of the sums is
// allowed (the bfloat16 mode).  With S the state before the eight, G_j the product of the decays up to token j and D_ji
// the product of those behind i up to j,
//     u_j = beta_j (v_j - G_j S^T k_j - sum_(i<j) D_ji (k_i . k_j) u_i)
//     o_j = G_j S^T q_j + sum_(i<=j) D_ji (k_i . q_j) u_i
//     S  <- G_7 S + sum_i D_7i k_i u_i
// so the sixteen products with S are independent of one another (one round of shuffles for all), and only the short
// triangular sums follow in order.  The coefficients, which the columns share, are made by delta_chunk_prep_kernel.  float32.
#include "common.cuh"

#define DL_THREADS 128
#define DL_ROWS 32
#define DL_TILE 16
#define DL_PREP_TOKENS 4

struct DeltaArgs {
    const float* x;                 // [T, ld] the packed float32 projection
    int T, prep_tokens, ld, q_off, k_off, v_off, b_off;
    const float* a;                 // decay projection (before the bias): [T, nh * d], or head_decay [T, nh]; rows a_ld apart
    int a_ld, head_decay;
    int nh, nkv, d, dv, taps;
    const float *conv_q, *conv_k, *conv_v;      // [channels, taps]
    const float *a_log, *dt_bias;               // [nh], [nh * d] or [nh]
    float q_scale;
    float* state;                   // [slots, state_elems]: S [nh, dv, d], then the convolution's rows [taps - 1, C]
    long long state_elems;
    const int *slots, *cu_q, *token_pos, *token_seq, *seq_lens;
    float* qkv;                     // out [T, C] prepared q, k, v (C = 2 nkv d + nh dv)
    float* g;                       // out [T, nh * d] or [T, nh]
    float* beta;                    // out [T, nh]
    float* out;                     // [T, nh * dv]
};

__device__ __forceinline__ float silu_f(float v) { return v / (1.0f + expf(-v)); }

// The convolution of one channel at token t: the taps oldest first, one chain of fused multiply-adds, the same whether a
// row comes from the step or from the state.  KT > 0: the number of taps at compile time; a token that has all its
// earlier rows in the step itself (every token of a prompt but the first few) reads them with fixed offsets.
template <int KT>
__device__ __forceinline__ float conv_channel(const DeltaArgs& p, int t, int i_step, int pos, int c, int col, const float* __restrict__ taps,
                                              const float* __restrict__ conv_state, int C) {
    const int K = KT > 0 ? KT : p.taps;
    const float* xc = p.x + (size_t)t * p.ld + col;
    float y = 0.f;
    if (KT > 0 && i_step >= KT - 1) {
        float in[KT > 0 ? KT : 1], w[KT > 0 ? KT : 1];
#pragma unroll
        for (int j = 0; j < KT; j++) {
            in[j] = __ldg(xc - (ptrdiff_t)j * p.ld);
            w[j] = __ldg(taps + KT - 1 - j);
        }
#pragma unroll
        for (int j = KT - 1; j >= 0; j--) y = fmaf(w[j], in[j], y);
        return y;
    }
    if (KT > 0) {          // the first tokens of a step: rows from the state and from the step, all loads before the chain
        float in[KT > 0 ? KT : 1], w[KT > 0 ? KT : 1];
#pragma unroll
        for (int j = 0; j < KT; j++) {
            in[j] = 0.f;
            w[j] = __ldg(taps + KT - 1 - j);
            if (pos - j >= 0) in[j] = j <= i_step ? __ldg(xc - (ptrdiff_t)j * p.ld) : conv_state[(size_t)(KT - 1 - (j - i_step)) * C + c];
        }
#pragma unroll
        for (int j = KT - 1; j >= 0; j--)
            if (pos - j >= 0) y = fmaf(w[j], in[j], y);
        return y;
    }
    for (int j = K - 1; j >= 0; j--) {
        if (pos - j < 0) continue;
        const float in = j <= i_step ? xc[-(ptrdiff_t)j * p.ld] : conv_state[(size_t)(K - 1 - (j - i_step)) * C + c];
        y = fmaf(taps[K - 1 - j], in, y);
    }
    return y;
}

// silu of a convolved projection: the fast exponential and division (these values may be rounded to bfloat16 anyway)
__device__ __forceinline__ float silu_fast(float v) { return __fdividef(v, 1.0f + __expf(-v)); }

// grid (tokens, units), 256 threads.  A unit is a group of query or key heads (convolution, silu, unit vectors; as many
// heads as fit 256 threads, a head of more than 256 channels alone), a piece of 1024 value channels (convolution, silu),
// a piece of 1024 decay channels, or the write strengths of all heads.
__device__ __forceinline__ int delta_heads_per_block(int d) { return d > 256 ? 1 : 256 / ((d + 31) / 32 * 32); }

template <int KT>
__global__ void __launch_bounds__(256) delta_prep_kernel(DeltaArgs p) {
    pdl_grid_sync();
    __shared__ float scratch[32];
    __shared__ float warp_ss[8];
    const int unit = blockIdx.y;
    // in a long step a block takes DL_PREP_TOKENS tokens in turn (one in a short step): the look-ups at the start of a token are a chain of dependent loads,
    // which a block of one token would spend most of its life on
#pragma unroll 1
    for (int t = blockIdx.x * p.prep_tokens; t < min(p.T, (int)(blockIdx.x + 1) * p.prep_tokens); t++) {
    __syncthreads();
    const int seq = p.token_seq[t], pos = p.token_pos[t];
    const int i_step = t - p.cu_q[seq];            // the token's place among the step's tokens of its sequence
    const int d = p.d, nq = p.nkv * d, nv = p.nh * p.dv, ng = p.head_decay ? p.nh : p.nh * d, C = 2 * nq + nv, K = p.taps;
    const float* conv_state = p.state + (size_t)p.slots[seq] * p.state_elems + (size_t)p.nh * d * p.dv;
    float* dst = p.qkv + (size_t)t * C;
    const int hpb = delta_heads_per_block(d), qk_units = (2 * p.nkv + hpb - 1) / hpb;
    const int v_units = (nv + 1023) / 1024, g_units = (ng + 1023) / 1024;
    if (unit < qk_units && d <= 256) {
        // thread -> (head of the unit, channel); a head's sum of squares: its warps' sums added in order
        const int dth = (d + 31) / 32 * 32, hl = threadIdx.x / dth, i = threadIdx.x % dth;
        const int head = unit * hpb + hl;           // 0 .. nkv - 1 query heads, then the key heads
        const bool live = hl < hpb && head < 2 * p.nkv && i < d;
        const bool is_q = head < p.nkv;
        const int hh = is_q ? head : head - p.nkv;
        float v = 0.f;
        if (live)
            v = silu_fast(conv_channel<KT>(p, t, i_step, pos, head * d + i, (is_q ? p.q_off : p.k_off) + hh * d + i,
                                    (is_q ? p.conv_q : p.conv_k) + ((size_t)hh * d + i) * K, conv_state, C));
        const float ws = warp_sum(v * v);
        if ((threadIdx.x & 31) == 0) warp_ss[threadIdx.x >> 5] = ws;
        __syncthreads();
        if (live) {
            float ss = 0.f;
            for (int w = hl * (dth / 32); w < (hl + 1) * (dth / 32); w++) ss += warp_ss[w];
            dst[head * d + i] = v * ((1.0f / sqrtf(ss + 1e-6f)) * (is_q ? p.q_scale : 1.0f));
        }
    } else if (unit < qk_units) {
        const bool is_q = unit < p.nkv;
        const int hh = is_q ? unit : unit - p.nkv;
        const float* taps = (is_q ? p.conv_q : p.conv_k) + (size_t)hh * d * K;
        const int c0 = unit * d, col0 = (is_q ? p.q_off : p.k_off) + hh * d;
        float v[2], ss = 0.f;                       // up to 512 channels per head
#pragma unroll
        for (int r = 0; r < 2; r++) {
            const int i = threadIdx.x + r * 256;
            v[r] = 0.f;
            if (i < d) {
                v[r] = silu_fast(conv_channel<KT>(p, t, i_step, pos, c0 + i, col0 + i, taps + (size_t)i * K, conv_state, C));
                ss = fmaf(v[r], v[r], ss);
            }
        }
        ss = block_sum(ss, scratch);
        const float inv = (1.0f / sqrtf(ss + 1e-6f)) * (is_q ? p.q_scale : 1.0f);
#pragma unroll
        for (int r = 0; r < 2; r++) {
            const int i = threadIdx.x + r * 256;
            if (i < d) dst[c0 + i] = v[r] * inv;
        }
    } else if (unit < qk_units + v_units) {
        float y[4];
#pragma unroll
        for (int r = 0; r < 4; r++) {
            const int c = (unit - qk_units) * 1024 + r * 256 + threadIdx.x;
            y[r] = c < nv ? conv_channel<KT>(p, t, i_step, pos, 2 * nq + c, p.v_off + c, p.conv_v + (size_t)c * K, conv_state, C) : 0.f;
        }
#pragma unroll
        for (int r = 0; r < 4; r++) {
            const int c = (unit - qk_units) * 1024 + r * 256 + threadIdx.x;
            if (c < nv) dst[2 * nq + c] = silu_fast(y[r]);
        }
    } else if (unit < qk_units + v_units + g_units) {
#pragma unroll
        for (int r = 0; r < 4; r++) {
            const int c = (unit - qk_units - v_units) * 1024 + r * 256 + threadIdx.x;
            if (c < ng) {
                const float z = p.a[(size_t)t * p.a_ld + c] + p.dt_bias[c];
                const float sp = z > 20.f ? z : log1pf(expf(z));
                p.g[(size_t)t * ng + c] = expf(-expf(p.a_log[p.head_decay ? c : c / d]) * sp);
            }
        }
    } else {
        for (int h = threadIdx.x; h < p.nh; h += blockDim.x) p.beta[(size_t)t * p.nh + h] = 1.0f / (1.0f + expf(-p.x[(size_t)t * p.ld + p.b_off + h]));
    }
    }
}

// The convolution's rows after the step: the raw projections of the sequence's last taps - 1 positions (zeros for
// positions before its start).  A thread owns a channel and goes through the rows in ascending order, so that a
// row kept from before the step is read before it is overwritten.
__global__ void conv_state_kernel(DeltaArgs p) {
    pdl_grid_sync();
    const int b = blockIdx.y;
    const int nq = p.nkv * p.d, nv = p.nh * p.dv, C = 2 * nq + nv, K = p.taps;
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= C) return;
    const int col = c < nq ? p.q_off + c : c < 2 * nq ? p.k_off + c - nq : p.v_off + c - 2 * nq;
    const int first = p.cu_q[b], n = p.cu_q[b + 1] - first;
    const int len = p.seq_lens[b], past = len - n;
    float* cs = p.state + (size_t)p.slots[b] * p.state_elems + (size_t)p.nh * p.d * p.dv;
    for (int r = 0; r < K - 1; r++) {
        const int pos = len - (K - 1) + r;
        float v = 0.f;
        if (pos >= past) v = p.x[(size_t)(first + pos - past) * p.ld + col];
        else if (pos >= 0) v = cs[(size_t)(r + n) * C + c];
        cs[(size_t)r * C + c] = v;
    }
}

// grid (column groups, heads, sequences); L lanes per column, DL_THREADS / L columns per block.  A thread's 32 rows are
// the quads 4 (l + L r) .. + 3 for r = 0..7, so that its q, k and g come as 16-byte reads of shared memory that the
// lanes of a column make side by side; rows beyond d are padding (k = q = 0, so their state stays 0).  The two dot
// products run as four chains each.
__device__ __forceinline__ void dl_cp16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src));
}
__device__ __forceinline__ void dl_cp4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src));
}

// HEAD: one decay per head and token (a number per token in shared memory).  It is then taken out of the first dot product,
// S^T k of the decayed state = g (S^T k), and the state is decayed while that product is being added over the lanes.
template <int L, int ROWS, bool HEAD>
__global__ void __launch_bounds__(DL_THREADS) delta_scan_kernel(DeltaArgs p) {
    pdl_grid_sync();
    extern __shared__ __align__(16) float sm[];
    constexpr int COLS = DL_THREADS / L, DPAD = ROWS * L;
    const int b = blockIdx.z, h = blockIdx.y, hk = h / (p.nh / p.nkv);
    const int d = p.d, dv = p.dv;
    const int l = threadIdx.x % L, jc = threadIdx.x / L;
    const int j = blockIdx.x * COLS + jc;           // the thread's column
    const bool live = j < dv;
    const int first = p.cu_q[b], n = p.cu_q[b + 1] - first;
    const int nq = p.nkv * d, C = 2 * nq + p.nh * dv;
    float* S_col = p.state + (size_t)p.slots[b] * p.state_elems + ((size_t)h * dv + (live ? j : 0)) * d;
    float S[ROWS];
#pragma unroll
    for (int r = 0; r < ROWS; r++) {
        const int i = 4 * (l + L * (r >> 2)) + (r & 3);
        S[r] = (live && i < d) ? S_col[i] : 0.f;
    }
    // Two buffers of a tile of tokens in shared memory: q, k, g [tile, DPAD] each (HEAD: g [tile]), v [tile, COLS], beta [tile].  The next
    // tile is on its way (cp.async) while this one is computed.  The padding rows beyond d are written once.
    constexpr int GW = HEAD ? 1 : DPAD;
    constexpr int BUF = DL_TILE * (2 * DPAD + GW + COLS + 1);
    const int j0 = blockIdx.x * COLS;
    const float* __restrict__ qkv = p.qkv;
    const float* __restrict__ gg = p.g;
    float* __restrict__ out = p.out;
    if (d < DPAD)
        for (int e = threadIdx.x; e < 2 * DL_TILE * (DPAD - d); e += DL_THREADS) {
            const int bb = e / (DL_TILE * (DPAD - d)), r = e % (DL_TILE * (DPAD - d));
            const int at = (r / (DPAD - d)) * DPAD + d + r % (DPAD - d);
            sm[bb * BUF + at] = 0.f;
            sm[bb * BUF + DL_TILE * DPAD + at] = 0.f;
            if (!HEAD) sm[bb * BUF + 2 * DL_TILE * DPAD + at] = 1.f;
        }
    const bool wide = (d & 3) == 0 && (C & 3) == 0;          // rows of q, k and the decay start on 16-byte boundaries
    auto stage = [&](int buf, int t0) {
        float* sq = sm + buf * BUF;
        float* sk = sq + DL_TILE * DPAD;
        float* sg = sk + DL_TILE * DPAD;
        float* sv = sg + DL_TILE * GW;
        float* sb = sv + DL_TILE * COLS;
        const int nt = min(DL_TILE, n - t0);
        if (HEAD)
            for (int e = threadIdx.x; e < nt; e += DL_THREADS) dl_cp4(sg + e, gg + (size_t)(first + t0 + e) * p.nh + h);
        if (wide) {
            const int per_row = d >> 2;
            for (int e = threadIdx.x; e < nt * per_row; e += DL_THREADS) {
                const int tt = e / per_row, i = (e - tt * per_row) * 4;
                const size_t t = (size_t)(first + t0 + tt);
                dl_cp16(sq + tt * DPAD + i, qkv + t * C + (size_t)hk * d + i);
                dl_cp16(sk + tt * DPAD + i, qkv + t * C + nq + (size_t)hk * d + i);
                if (!HEAD) dl_cp16(sg + tt * DPAD + i, gg + t * p.nh * d + (size_t)h * d + i);
            }
        } else {
            for (int e = threadIdx.x; e < nt * d; e += DL_THREADS) {
                const int tt = e / d, i = e - tt * d;
                const size_t t = (size_t)(first + t0 + tt);
                dl_cp4(sq + tt * DPAD + i, qkv + t * C + (size_t)hk * d + i);
                dl_cp4(sk + tt * DPAD + i, qkv + t * C + nq + (size_t)hk * d + i);
                if (!HEAD) dl_cp4(sg + tt * DPAD + i, gg + t * p.nh * d + (size_t)h * d + i);
            }
        }
        for (int e = threadIdx.x; e < nt * COLS; e += DL_THREADS) {
            const int tt = e / COLS, c = e - tt * COLS;
            if (j0 + c < dv) dl_cp4(sv + e, qkv + (size_t)(first + t0 + tt) * C + 2 * nq + (size_t)h * dv + j0 + c);
        }
        for (int e = threadIdx.x; e < nt; e += DL_THREADS) dl_cp4(sb + e, p.beta + (size_t)(first + t0 + e) * p.nh + h);
    };
    if (n > 0) stage(0, 0);
    asm volatile("cp.async.commit_group;\n" ::);
    for (int t0 = 0, it = 0; t0 < n; t0 += DL_TILE, it++) {
        const int nt = min(DL_TILE, n - t0);
        if (t0 + DL_TILE < n) stage((it + 1) & 1, t0 + DL_TILE);
        asm volatile("cp.async.commit_group;\n" ::);
        asm volatile("cp.async.wait_group 1;\n" ::);
        __syncthreads();
        const float* sq = sm + (it & 1) * BUF;
        const float* sk = sq + DL_TILE * DPAD;
        const float* sg = sk + DL_TILE * DPAD;
        const float* sv = sg + DL_TILE * GW;
        const float* sb = sv + DL_TILE * COLS;
        for (int tt = 0; tt < nt; tt++) {
            const float4* q4 = reinterpret_cast<const float4*>(sq + tt * DPAD);
            const float4* k4 = reinterpret_cast<const float4*>(sk + tt * DPAD);
            const float4* g4 = reinterpret_cast<const float4*>(sg + tt * DPAD);
            float4 kk[ROWS / 4], qq[ROWS / 4];
            float a0 = 0.f, a1 = 0.f, a2 = 0.f, a3 = 0.f;
#pragma unroll
            for (int r = 0; r < ROWS / 4; r++) {
                kk[r] = k4[l + L * r];
                qq[r] = q4[l + L * r];           // read now, used after the first reduction
            }
            const float gh = HEAD ? sg[tt] : 1.f;
#pragma unroll
            for (int r = 0; r < ROWS / 4; r++) {
                if (!HEAD) {
                    const float4 g = g4[l + L * r];
                    S[4 * r] *= g.x;
                    S[4 * r + 1] *= g.y;
                    S[4 * r + 2] *= g.z;
                    S[4 * r + 3] *= g.w;
                }
                a0 = fmaf(kk[r].x, S[4 * r], a0);
                a1 = fmaf(kk[r].y, S[4 * r + 1], a1);
                a2 = fmaf(kk[r].z, S[4 * r + 2], a2);
                a3 = fmaf(kk[r].w, S[4 * r + 3], a3);
            }
            float acc = (a0 + a1) + (a2 + a3);
#pragma unroll
            for (int o = L / 2; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
            if (HEAD) {
#pragma unroll
                for (int r = 0; r < ROWS; r++) S[r] *= gh;
                acc *= gh;
            }
            const float u = sb[tt] * (sv[tt * COLS + jc] - acc);
            a0 = a1 = a2 = a3 = 0.f;
#pragma unroll
            for (int r = 0; r < ROWS / 4; r++) {
                const float4 q = qq[r];
                S[4 * r] = fmaf(kk[r].x, u, S[4 * r]);
                S[4 * r + 1] = fmaf(kk[r].y, u, S[4 * r + 1]);
                S[4 * r + 2] = fmaf(kk[r].z, u, S[4 * r + 2]);
                S[4 * r + 3] = fmaf(kk[r].w, u, S[4 * r + 3]);
                a0 = fmaf(q.x, S[4 * r], a0);
                a1 = fmaf(q.y, S[4 * r + 1], a1);
                a2 = fmaf(q.z, S[4 * r + 2], a2);
                a3 = fmaf(q.w, S[4 * r + 3], a3);
            }
            float oacc = (a0 + a1) + (a2 + a3);
#pragma unroll
            for (int o = L / 2; o > 0; o >>= 1) oacc += __shfl_xor_sync(0xffffffffu, oacc, o);
            if (live && l == 0) out[(size_t)(first + t0 + tt) * p.nh * dv + (size_t)h * dv + j] = oacc;
        }
        __syncthreads();          // the tile after the next one goes into this buffer
    }
    if (live) {
#pragma unroll
        for (int r = 0; r < ROWS; r++) {
            const int i = 4 * (l + L * (r >> 2)) + (r & 3);
            if (i < d) S_col[i] = S[r];
        }
    }
}

// ---- eight tokens at a time

#define DC 8                       // tokens per chunk
#define DC_REC (4 * DC + 2 * DC * DC)      // floats per (chunk, head): beta, beta G, G, D_7i, then M[j][i] and P[j][i]

// Chunk c of the step's sequence b has its record at slot cu_q[b] / DC + b + c (distinct for all chunks of a step).
__device__ __forceinline__ int dc_slot(int first, int b, int c) { return first / DC + b + c; }

// grid (chunks of the longest sequence, query/key heads, sequences), 128 threads: the products k_i . k_j and k_i . q_j of a
// chunk, then the records of the value heads that share the keys.  Tokens beyond the sequence's end count as k = q = 0,
// g = 1, beta = 0.
__global__ void __launch_bounds__(128) delta_chunk_prep_kernel(DeltaArgs p, float* __restrict__ rec) {
    pdl_grid_sync();
    extern __shared__ float sm[];            // k [DC][d], q [DC][d]
    __shared__ float kk[DC][DC], kq[DC][DC];
    const int c = blockIdx.x, hk = blockIdx.y, b = blockIdx.z;
    const int first = p.cu_q[b], n = p.cu_q[b + 1] - first, t0 = c * DC;
    if (t0 >= n) return;
    const int nt = min(DC, n - t0), d = p.d, nq = p.nkv * d, C = 2 * nq + p.nh * p.dv;
    float *sk = sm, *sq = sm + DC * d;
    for (int e = threadIdx.x; e < DC * d; e += 128) {
        const int j = e / d, i = e - j * d;
        const float* row = p.qkv + (size_t)(first + t0 + j) * C + (size_t)hk * d + i;
        sq[e] = j < nt ? row[0] : 0.f;
        sk[e] = j < nt ? row[nq] : 0.f;
    }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int e = warp; e < 2 * DC * DC; e += 4) {
        const int j = (e / DC) % DC, i = e % DC;
        const bool with_q = e >= DC * DC;
        if (i > j || (!with_q && i == j)) continue;          // uniform over the warp
        const float *a = sk + i * d, *bb = (with_q ? sq : sk) + j * d;
        float s = 0.f;
        for (int x = lane; x < d; x += 32) s = fmaf(a[x], bb[x], s);
        s = warp_sum(s);
        if (lane == 0) (with_q ? kq : kk)[j][i] = s;
    }
    __syncthreads();
    const int share = p.nh / p.nkv;
    for (int e = threadIdx.x; e < share * DC; e += 128) {
        const int h = hk * share + e / DC, j = e % DC;
        float g[DC];
#pragma unroll
        for (int i = 0; i < DC; i++) g[i] = i < nt ? p.g[(size_t)(first + t0 + i) * p.nh + h] : 1.f;
        const float beta = j < nt ? p.beta[(size_t)(first + t0 + j) * p.nh + h] : 0.f;
        float G = 1.f, E = 1.f;
#pragma unroll
        for (int i = 0; i < DC; i++) {
            if (i <= j) G *= g[i];
            if (i > j) E *= g[i];
        }
        float* r = rec + ((size_t)dc_slot(first, b, c) * p.nh + h) * DC_REC;
        r[j] = beta;
        r[DC + j] = beta * G;
        r[2 * DC + j] = G;
        r[3 * DC + j] = E;
        float D = 1.f;
#pragma unroll
        for (int i = DC - 1; i >= 0; i--) {          // D_ji, from i = j down
            const bool in = i <= j;
            r[4 * DC + j * DC + i] = i < j ? beta * D * (i + 1 <= j ? g[i + 1 < DC ? i + 1 : DC - 1] : 1.f) * kk[j][i] : 0.f;
            if (i < j) D *= g[i + 1 < DC ? i + 1 : DC - 1];
            r[4 * DC + DC * DC + j * DC + i] = in ? D * kq[j][i] : 0.f;
        }
    }
}

__device__ __forceinline__ unsigned long long dl_pack(float lo, float hi) {
    unsigned long long r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ void dl_unpack(unsigned long long v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ unsigned long long dl_fma2(unsigned long long a, unsigned long long b, unsigned long long c) {
    unsigned long long r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ unsigned long long dl_mul2(unsigned long long a, unsigned long long b) {
    unsigned long long r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}

// The layout of delta_scan_kernel: grid (column groups, heads, sequences), L lanes per column, a thread's ROWS rows the quads
// 4 (l + L r) .. + 3, held as pairs for the two-at-a-time float32 instructions.
template <int L, int ROWS>
__global__ void __launch_bounds__(DL_THREADS) delta_chunk_scan_kernel(DeltaArgs p, const float* __restrict__ rec) {
    pdl_grid_sync();
    extern __shared__ __align__(16) float sm[];
    constexpr int COLS = DL_THREADS / L, DPAD = ROWS * L, CHUNKS = DL_TILE / DC, Q4 = ROWS / 4;
    const int b = blockIdx.z, h = blockIdx.y, hk = h / (p.nh / p.nkv);
    const int d = p.d, dv = p.dv;
    const int l = threadIdx.x % L, jc = threadIdx.x / L;
    const int col = blockIdx.x * COLS + jc;
    const bool live = col < dv;
    const int first = p.cu_q[b], n = p.cu_q[b + 1] - first;
    const int nq = p.nkv * d, C = 2 * nq + p.nh * dv;
    float* S_col = p.state + (size_t)p.slots[b] * p.state_elems + ((size_t)h * dv + (live ? col : 0)) * d;
    unsigned long long S[ROWS / 2];
#pragma unroll
    for (int r = 0; r < ROWS / 2; r++) {
        const int i = 4 * (l + L * (r >> 1)) + 2 * (r & 1);
        S[r] = dl_pack(live && i < d ? S_col[i] : 0.f, live && i + 1 < d ? S_col[i + 1] : 0.f);
    }
    // two buffers of a tile: q, k [tile, DPAD], the chunks' records, v [tile, COLS]
    constexpr int BUF = DL_TILE * (2 * DPAD + COLS) + CHUNKS * DC_REC;
    const int j0 = blockIdx.x * COLS;
    const float* __restrict__ qkv = p.qkv;
    float* __restrict__ out = p.out;
    if (d < DPAD)
        for (int e = threadIdx.x; e < 2 * 2 * DL_TILE * (DPAD - d); e += DL_THREADS) {
            const int bb = e / (2 * DL_TILE * (DPAD - d)), r = e % (2 * DL_TILE * (DPAD - d));
            sm[bb * BUF + (r / (DPAD - d)) * DPAD + d + r % (DPAD - d)] = 0.f;
        }
    const bool wide = (d & 3) == 0 && (C & 3) == 0;
    // a thread's first piece of a tile's rows and the step to its next one, so that staging divides nothing
    const int per_row = wide ? d >> 2 : d, piece = wide ? 4 : 1;
    const int tt_first = threadIdx.x / per_row, i_first = threadIdx.x % per_row, tt_step = DL_THREADS / per_row, i_step = DL_THREADS % per_row;
    auto stage = [&](int buf, int t0) {
        float* sq = sm + buf * BUF;
        float* sk = sq + DL_TILE * DPAD;
        float* sr = sk + DL_TILE * DPAD;
        float* sv = sr + CHUNKS * DC_REC;
        const int nt = min(DL_TILE, n - t0), nc = (nt + DC - 1) / DC, np = nc * DC;        // np: with the last chunk's missing tokens
        const float* base = qkv + (size_t)(first + t0) * C + (size_t)hk * d;
        for (int tt = tt_first, ip = i_first; tt < np;) {
            const int i = ip * piece;
            float *dq = sq + tt * DPAD + i, *dk = sk + tt * DPAD + i;
            const float* row = base + (size_t)tt * C + i;
            if (wide) {
                if (tt < nt) {
                    dl_cp16(dq, row);
                    dl_cp16(dk, row + nq);
                } else {
                    *reinterpret_cast<float4*>(dq) = make_float4(0.f, 0.f, 0.f, 0.f);
                    *reinterpret_cast<float4*>(dk) = make_float4(0.f, 0.f, 0.f, 0.f);
                }
            } else if (tt < nt) {
                dl_cp4(dq, row);
                dl_cp4(dk, row + nq);
            } else {
                *dq = 0.f;
                *dk = 0.f;
            }
            tt += tt_step;
            ip += i_step;
            if (ip >= per_row) {
                ip -= per_row;
                tt++;
            }
        }
        for (int e = threadIdx.x; e < nc * (DC_REC / 4); e += DL_THREADS) {
            const int cc = e / (DC_REC / 4), x = (e - cc * (DC_REC / 4)) * 4;
            dl_cp16(sr + cc * DC_REC + x, rec + ((size_t)dc_slot(first, b, t0 / DC + cc) * p.nh + h) * DC_REC + x);
        }
        for (int e = threadIdx.x; e < np * COLS; e += DL_THREADS) {
            const int tt = e / COLS, c = e - tt * COLS;
            if (tt < nt && j0 + c < dv) dl_cp4(sv + e, qkv + (size_t)(first + t0 + tt) * C + 2 * nq + (size_t)h * dv + j0 + c);
            else sv[e] = 0.f;
        }
    };
    if (n > 0) stage(0, 0);
    asm volatile("cp.async.commit_group;\n" ::);
    for (int t0 = 0, it = 0; t0 < n; t0 += DL_TILE, it++) {
        const int nt = min(DL_TILE, n - t0);
        if (t0 + DL_TILE < n) stage((it + 1) & 1, t0 + DL_TILE);
        asm volatile("cp.async.commit_group;\n" ::);
        asm volatile("cp.async.wait_group 1;\n" ::);
        __syncthreads();
        const float* sq = sm + (it & 1) * BUF;
        const float* sk = sq + DL_TILE * DPAD;
        const float* sr = sk + DL_TILE * DPAD;
        const float* sv = sr + CHUNKS * DC_REC;
#pragma unroll 1
        for (int c0 = 0; c0 < nt; c0 += DC) {
            const ulonglong2* k2 = reinterpret_cast<const ulonglong2*>(sk + c0 * DPAD) + l;
            const ulonglong2* q2 = reinterpret_cast<const ulonglong2*>(sq + c0 * DPAD) + l;
            const float4* r4 = reinterpret_cast<const float4*>(sr + (c0 / DC) * DC_REC);
            // S^T k_j and S^T q_j of all eight tokens
            unsigned long long ak[DC], aq[DC];
#pragma unroll
            for (int j = 0; j < DC; j++) ak[j] = aq[j] = 0ull;
#pragma unroll
            for (int r = 0; r < Q4; r++) {
#pragma unroll
                for (int j = 0; j < DC; j++) {
                    const ulonglong2 kv = k2[j * (DPAD / 4) + L * r], qv = q2[j * (DPAD / 4) + L * r];
                    ak[j] = dl_fma2(kv.y, S[2 * r + 1], dl_fma2(kv.x, S[2 * r], ak[j]));
                    aq[j] = dl_fma2(qv.y, S[2 * r + 1], dl_fma2(qv.x, S[2 * r], aq[j]));
                }
            }
            float A[DC], O[DC];
#pragma unroll
            for (int j = 0; j < DC; j++) {
                float lo, hi;
                dl_unpack(ak[j], lo, hi);
                A[j] = lo + hi;
                dl_unpack(aq[j], lo, hi);
                O[j] = lo + hi;
            }
#pragma unroll
            for (int o = L / 2; o > 0; o >>= 1)
#pragma unroll
                for (int j = 0; j < DC; j++) {
                    A[j] += __shfl_xor_sync(0xffffffffu, A[j], o);
                    O[j] += __shfl_xor_sync(0xffffffffu, O[j], o);
                }
            // the triangular sums
            float u[DC];
            float bv[DC], bg[DC], gg[DC];
#pragma unroll
            for (int x = 0; x < DC / 4; x++) {
                const float4 t1 = r4[x], t2 = r4[DC / 4 + x], t3 = r4[2 * (DC / 4) + x];
                bv[4 * x] = t1.x, bv[4 * x + 1] = t1.y, bv[4 * x + 2] = t1.z, bv[4 * x + 3] = t1.w;
                bg[4 * x] = t2.x, bg[4 * x + 1] = t2.y, bg[4 * x + 2] = t2.z, bg[4 * x + 3] = t2.w;
                gg[4 * x] = t3.x, gg[4 * x + 1] = t3.y, gg[4 * x + 2] = t3.z, gg[4 * x + 3] = t3.w;
            }
#pragma unroll
            for (int j = 0; j < DC; j++) {
                float m[DC], pr[DC];
#pragma unroll
                for (int x = 0; x < DC / 4; x++) {
                    const float4 t1 = r4[DC + j * (DC / 4) + x], t2 = r4[DC + DC * DC / 4 + j * (DC / 4) + x];
                    m[4 * x] = t1.x, m[4 * x + 1] = t1.y, m[4 * x + 2] = t1.z, m[4 * x + 3] = t1.w;
                    pr[4 * x] = t2.x, pr[4 * x + 1] = t2.y, pr[4 * x + 2] = t2.z, pr[4 * x + 3] = t2.w;
                }
                float v = fmaf(-bg[j], A[j], bv[j] * sv[(c0 + j) * COLS + jc]);
#pragma unroll
                for (int i = 0; i < j; i++) v = fmaf(-m[i], u[i], v);
                u[j] = v;
                float o = gg[j] * O[j];
#pragma unroll
                for (int i = 0; i <= j; i++) o = fmaf(pr[i], u[i], o);
                O[j] = o;
            }
            // every lane of a column has all of them: lane l stores token j0 + l
            constexpr int LS = L < DC ? L : DC;
#pragma unroll
            for (int j0 = 0; j0 < DC; j0 += LS) {
                float o = O[j0];
#pragma unroll
                for (int k = 1; k < LS; k++) o = l == k ? O[j0 + k] : o;
                if (live && l < LS && c0 + j0 + l < nt) out[(size_t)(first + t0 + c0 + j0 + l) * p.nh * dv + (size_t)h * dv + col] = o;
            }
            // the state behind the chunk; long columns read the keys a second time instead of keeping them in registers
            if (ROWS > 8) asm volatile("" ::: "memory");
            const unsigned long long g2 = dl_pack(gg[DC - 1], gg[DC - 1]);
            unsigned long long w2[DC];
#pragma unroll
            for (int x = 0; x < DC / 4; x++) {
                const float4 t1 = r4[3 * (DC / 4) + x];
                const float e4[4] = {t1.x, t1.y, t1.z, t1.w};
#pragma unroll
                for (int y = 0; y < 4; y++) {
                    const float w = e4[y] * u[4 * x + y];
                    w2[4 * x + y] = dl_pack(w, w);
                }
            }
#pragma unroll
            for (int r = 0; r < Q4; r++) {
                unsigned long long s0 = dl_mul2(S[2 * r], g2), s1 = dl_mul2(S[2 * r + 1], g2);
#pragma unroll
                for (int j = 0; j < DC; j++) {
                    const ulonglong2 kv = k2[j * (DPAD / 4) + L * r];
                    s0 = dl_fma2(kv.x, w2[j], s0);
                    s1 = dl_fma2(kv.y, w2[j], s1);
                }
                S[2 * r] = s0;
                S[2 * r + 1] = s1;
            }
        }
        __syncthreads();          // the tile after the next one goes into this buffer
    }
    if (live) {
#pragma unroll
        for (int r = 0; r < ROWS / 2; r++) {
            const int i = 4 * (l + L * (r >> 1)) + 2 * (r & 1);
            float lo, hi;
            dl_unpack(S[r], lo, hi);
            if (i < d) S_col[i] = lo;
            if (i + 1 < d) S_col[i + 1] = hi;
        }
    }
}

// floats of scratch for the chunks' records of a step
extern "C" long long illm_delta_chunk_scratch(int T, int B, int nh) { return ((long long)T / DC + B + 1) * nh * DC_REC; }

extern "C" int illm_delta_rule_supported(int d, int dv, int taps) { return d >= 1 && d <= 16 * DL_ROWS && dv >= 1 && taps >= 1 && taps <= 64; }

template <int L, int ROWS, bool HEAD>
static void launch_scan_as(const DeltaArgs& p, int B, int n_sms, cudaStream_t s) {
    constexpr int COLS = DL_THREADS / L;
    size_t smem = (size_t)(2 * DL_TILE * (2 * ROWS * L + (HEAD ? 1 : ROWS * L) + COLS + 1)) * sizeof(float);
    // The scan is bound by what an SM's shared memory delivers per clock, so its blocks must spread over the SMs.  Launched
    // behind kernels that still hold most SMs, a small grid would be packed onto the few SMs that are free first (measured: 32
    // blocks, 2.5 ms instead of 0.95 ms).  Asking for more shared memory than the tiles need caps the blocks per SM at what an
    // even spread gives.
    const long long blocks = (long long)((p.dv + COLS - 1) / COLS) * p.nh * B;
    const long long per_sm = (blocks + n_sms - 1) / n_sms;
    if (per_sm < 5) {
        const size_t spread = (size_t)(220 * 1024) / (size_t)per_sm - 2048;
        smem = smem > spread ? smem : (spread < (size_t)200 * 1024 ? spread : (size_t)200 * 1024);
    }
    static bool raised = false;
    if (!raised) {
        cudaFuncSetAttribute(delta_scan_kernel<L, ROWS, HEAD>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        raised = true;
    }
    illm_launch(delta_scan_kernel<L, ROWS, HEAD>, dim3((p.dv + COLS - 1) / COLS, p.nh, B), dim3(DL_THREADS), smem, s, p);
}

template <int L, int ROWS>
static void launch_scan(const DeltaArgs& p, int B, int n_sms, cudaStream_t s, const float* rec) {
    if constexpr (ROWS <= 16) if (rec) {        // (eight tokens at a time with 32 rows per thread do not fit the registers)
        constexpr int COLS = DL_THREADS / L;
        size_t smem = (size_t)2 * (DL_TILE * (2 * ROWS * L + COLS) + (DL_TILE / DC) * DC_REC) * sizeof(float);
        const long long blocks = (long long)((p.dv + COLS - 1) / COLS) * p.nh * B, per_sm = (blocks + n_sms - 1) / n_sms;
        if (per_sm < 5) {          // as for the scan above: an even spread over the SMs
            const size_t spread = (size_t)(220 * 1024) / (size_t)per_sm - 2048;
            smem = smem > spread ? smem : (spread < (size_t)200 * 1024 ? spread : (size_t)200 * 1024);
        }
        static bool raised = false;
        if (!raised) {
            cudaFuncSetAttribute(delta_chunk_scan_kernel<L, ROWS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
            raised = true;
        }
        illm_launch((delta_chunk_scan_kernel<L, ROWS>), dim3((p.dv + COLS - 1) / COLS, p.nh, B), dim3(DL_THREADS), smem, s, p, rec);
        return;
    }
    if (p.head_decay) launch_scan_as<L, ROWS, true>(p, B, n_sms, s);
    else launch_scan_as<L, ROWS, false>(p, B, n_sms, s);
}

// A column's rows over L lanes of 32 rows each, or, while the grid of ONE sequence then still fits the SMs once, over 2 L
// lanes of 16 rows or 4 L lanes of 8: a sequence's tokens are a chain, and fewer rows per thread shorten every link of it
// (one prompt of 2,048 tokens, 8 heads of 128 x 128: 0.78 / 0.62 ms with 32 / 16 rows; with two blocks on an SM the
// shorter rows gain nothing).  The choice does not depend on the batch, or a row's bits would.
template <int L>
static void launch_scan_for(const DeltaArgs& p, int B, cudaStream_t s, const float* rec) {
    static int n_sms = 0;
    if (!n_sms) {
        int dev = 0;
        cudaGetDevice(&dev);
        cudaDeviceGetAttribute(&n_sms, cudaDevAttrMultiProcessorCount, dev);
        if (n_sms <= 0) n_sms = 1;
    }
    constexpr int L2 = 2 * L <= 32 ? 2 * L : L, L4 = 4 * L <= 32 ? 4 * L : L2;
    auto blocks_of = [&](int lanes) { return (long long)((p.dv + DL_THREADS / lanes - 1) / (DL_THREADS / lanes)) * p.nh; };
    if (L4 != L2 && blocks_of(L4) <= n_sms) launch_scan<L4, 8>(p, B, n_sms, s, rec);
    else if (L2 != L && (rec || blocks_of(L2) <= n_sms)) launch_scan<L2, 16>(p, B, n_sms, s, rec);
    else launch_scan<L, 32>(p, B, n_sms, s, rec);
}

// x: [T, ld] float32 with q at q_off (nkv * d columns), k at k_off, v at v_off (nh * dv), beta's logits at b_off (nh).
// state: float32 [slots, state_elems], state_elems >= nh * d * dv + (taps - 1) * (2 nkv d + nh dv).
// a: the decay projection, rows a_ld apart: nh * d columns, or with head_decay nh.
// chunks (head_decay only; nullptr: token by token): illm_delta_chunk_scratch floats, the scan then takes eight tokens at a
// time; max_q the most tokens of one sequence.
// Scratch qkv [T, 2 nkv d + nh dv], g [T, nh d] (head_decay: [T, nh]), beta [T, nh]; out [T, nh dv].
extern "C" int illm_delta_rule(const float* x, int T, int ld, int q_off, int k_off, int v_off, int b_off, const float* a, int a_ld, int head_decay, int nh, int nkv, int d,
                               int dv, int taps, const float* conv_q, const float* conv_k, const float* conv_v, const float* a_log,
                               const float* dt_bias, float q_scale, float* state, long long state_elems, const int* slots, const int* cu_q,
                               const int* token_pos, const int* token_seq, const int* seq_lens, float* qkv, float* g, float* beta, float* out,
                               int B, int max_q, float* chunks, void* stream) {
    if (T <= 0 || B <= 0) return 0;
    if (!illm_delta_rule_supported(d, dv, taps) || nkv <= 0 || nh % nkv || a_ld < (head_decay ? nh : nh * d) || (chunks && (!head_decay || max_q <= 0 || nkv > 65535 || B > 65535))) return ILLM_ERR_BAD_ARG;
    const long long C = 2LL * nkv * d + (long long)nh * dv;
    if (state_elems < (long long)nh * d * dv + (taps - 1) * C) return ILLM_ERR_BAD_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    DeltaArgs p;
    p.x = x; p.T = T; p.ld = ld; p.q_off = q_off; p.k_off = k_off; p.v_off = v_off; p.b_off = b_off;
    p.a = a; p.a_ld = a_ld; p.head_decay = head_decay; p.nh = nh; p.nkv = nkv; p.d = d; p.dv = dv; p.taps = taps;
    p.conv_q = conv_q; p.conv_k = conv_k; p.conv_v = conv_v; p.a_log = a_log; p.dt_bias = dt_bias; p.q_scale = q_scale;
    p.state = state; p.state_elems = state_elems; p.slots = slots; p.cu_q = cu_q; p.token_pos = token_pos; p.token_seq = token_seq;
    p.seq_lens = seq_lens; p.qkv = qkv; p.g = g; p.beta = beta; p.out = out;
    const int hpb = d > 256 ? 1 : 256 / ((d + 31) / 32 * 32);
    const long long units = (2LL * nkv + hpb - 1) / hpb + ((long long)nh * dv + 1023) / 1024 + ((long long)nh * (head_decay ? 1 : d) + 1023) / 1024 + 1;
    if (units > 65535) return ILLM_ERR_BAD_ARG;
    p.prep_tokens = T >= 512 ? DL_PREP_TOKENS : 1;
    const dim3 pgrid((T + p.prep_tokens - 1) / p.prep_tokens, (unsigned)units);
    if (taps == 1) illm_launch(delta_prep_kernel<1>, pgrid, dim3(256), 0, s, p);
    else if (taps == 2) illm_launch(delta_prep_kernel<2>, pgrid, dim3(256), 0, s, p);
    else if (taps == 3) illm_launch(delta_prep_kernel<3>, pgrid, dim3(256), 0, s, p);
    else if (taps == 4) illm_launch(delta_prep_kernel<4>, pgrid, dim3(256), 0, s, p);
    else illm_launch(delta_prep_kernel<0>, pgrid, dim3(256), 0, s, p);
    if (taps > 1) illm_launch(conv_state_kernel, dim3((unsigned)((C + 127) / 128), B), dim3(128), 0, s, p);
    if (chunks) {
        const size_t smem = (size_t)2 * DC * d * sizeof(float);
        illm_launch(delta_chunk_prep_kernel, dim3((max_q + DC - 1) / DC, nkv, B), dim3(128), smem, s, p, chunks);
    }
    if (d <= 32) launch_scan_for<1>(p, B, s, chunks);
    else if (d <= 64) launch_scan_for<2>(p, B, s, chunks);
    else if (d <= 128) launch_scan_for<4>(p, B, s, chunks);
    else if (d <= 256) launch_scan_for<8>(p, B, s, chunks);
    else launch_scan_for<16>(p, B, s, chunks);
    return illm_launch_status();
}
