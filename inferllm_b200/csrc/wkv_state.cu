// A time-mixing recurrence with a decay per head and key channel that every token makes itself, and a bonus for the token's
// own contribution:
//
//   o_t = S_(t-1)^T r_t + (r_t . (u * k_t)) v_t        (S: [d, dv] float32 per sequence and head)
//   S_t = diag(w_t) S_(t-1) + k_t v_t^T
//
// r, k, w are rows of d channels per head, v of dv.  The state lives in the cache's per-sequence storage, column by column
// ([slots, heads, dv, d] float32), so that a thread's rows are 16-byte pieces; a step loads it, runs its tokens in order and
// stores it.  Everything here is float32, in the float32 mode and in the bfloat16 mode alike.
//
// token_mix_kernel       several blends of a token's row and the row before it, x + (x' - x) * mu_s, each rounded once to the
//                        compute dtype as the input of its own matrix product; the row before a step's first token is
//                        per-sequence state (zeros when a sequence starts)
// token_mix_state_kernel the sequences' last rows into that state (steps of several tokens; a step of one token per sequence
//                        does it in the first kernel)
// wkv_prep_kernel        w = exp(-exp(w2 tanh(z) + w0)) from the inner products z of a low-rank map, and the bonus
//                        r . (u * k) per token and head
// wkv_scan_kernel        the recurrence token by token, for steps of any length (the float32 mode; short steps)
// wkv_chunk_prep_kernel, wkv_chunk_kernel
//                        the recurrence sixteen tokens at a time, for prompts in the bfloat16 mode (w2 in bfloat16)
// wkv_step_kernel        decay, bonus, recurrence, per-head unit norm and gate for one token per sequence in one kernel that
//                        also adds up the projections' K slices (the bfloat16 mode's decoding)
//
// wkv_scan_kernel: the columns of S never meet, so a block owns (sequence, head, a run of columns) and a thread keeps 16 rows
// of four columns in registers for the whole step, the rows of a column group over LI neighbouring lanes, as the scan with one
// decay per head does (decay_state.cu); here r, k and w of a token are three staged rows, and two rows of the state share one
// instruction (fma.rn.f32x2).
//
// Sixteen tokens at a time.  With the state S in front of a chunk, P_t the product of the decays of the chunk's tokens before
// t, Q_t that of those behind t, and P all of them (per key channel; products of decays are never divided by one another):
//
//   o_t = S^T (r_t * P_t) + sum over s <= t of A[t, s] v_s
//   A[t, s] = sum_i r_t,i k_s,i (product of w_i over the tokens between s and t),   A[t, t] = sum_i r_t,i u_i k_t,i
//   S <- diag(P) S + sum_s (k_s * Q_s) v_s^T
//
// wkv_chunk_prep_kernel makes w (the low-rank map's outer product on warp-level MMA, tanh as two bfloat16 terms), the scaled
// rows r_t * P_t and k_t * Q_t in place of r and k, A and P, a block per chunk and head; wkv_chunk_kernel runs the chunks with
// the state in registers: its products take one multiply-add per state element instead of three, and a chunk's tokens do
// not wait for one another.  A long prompt of few sequences is cut into segments that run side by side: pass 0 runs every
// segment but the last for its state alone, from zero (the first from the sequence's state), and leaves that state and the
// product of its decays; wkv_fold_kernel turns these into the states that the later segments start from, and pass 1 runs
// every segment in full.  The sums have another order than token by token, so the float32 mode never takes this form.
#include <type_traits>

#include "common.cuh"

typedef unsigned long long f2;      // two float32 in one 64-bit register

__device__ __forceinline__ f2 f2_pack(float lo, float hi) {
    f2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ void f2_unpack(f2 v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ f2 f2_fma(f2 a, f2 b, f2 c) {
    f2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ f2 f2_mul(f2 a, f2 b) {
    f2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}

__device__ __forceinline__ void wk_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void wk_store4(bf16* p, float4 v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&lo), *reinterpret_cast<const unsigned*>(&hi));
}

// ---- the blends

struct TokenMixArgs {
    const float* x;                 // [T, H]
    int H, n_mix;
    const float* mu;                // [n_mix, H]
    float* prev;                    // the slots' previous rows, prev_stride floats apart
    long long prev_stride;
    const int *slots, *cu_q, *token_seq;
    long long group_stride;         // elements from one blend's matrix to the next
    int single;                     // every sequence has one token: its row becomes the previous row here
};

template <typename TA, int V>
__global__ void __launch_bounds__(256) token_mix_kernel(TokenMixArgs a, TA* __restrict__ out) {
    pdl_grid_sync();
    const int t = blockIdx.x, c = (blockIdx.y * 256 + threadIdx.x) * V;
    if (c >= a.H) return;
    const int b = a.token_seq[t];
    const bool first = t == a.cu_q[b];
    float* pv = a.prev + (size_t)a.slots[b] * a.prev_stride;
    const float* xr = a.x + (size_t)t * a.H;
    const float* xp = first ? pv : xr - a.H;
    if (V == 4) {
        const float4 cur = *reinterpret_cast<const float4*>(xr + c), old = *reinterpret_cast<const float4*>(xp + c);
        if (a.single) *reinterpret_cast<float4*>(pv + c) = cur;
        for (int s = 0; s < a.n_mix; s++) {
            const float4 m = *reinterpret_cast<const float4*>(a.mu + (size_t)s * a.H + c);
            wk_store4(out + s * a.group_stride + (size_t)t * a.H + c,
                      make_float4(fmaf(old.x - cur.x, m.x, cur.x), fmaf(old.y - cur.y, m.y, cur.y), fmaf(old.z - cur.z, m.z, cur.z), fmaf(old.w - cur.w, m.w, cur.w)));
        }
    } else {
        const float cur = xr[c], old = xp[c];
        if (a.single) pv[c] = cur;
        for (int s = 0; s < a.n_mix; s++)
            out[s * a.group_stride + (size_t)t * a.H + c] = from_f32<TA>(fmaf(old - cur, a.mu[(size_t)s * a.H + c], cur));
    }
}

__global__ void token_mix_state_kernel(TokenMixArgs a) {
    pdl_grid_sync();
    const int b = blockIdx.x, n = a.cu_q[b + 1];
    if (n == a.cu_q[b]) return;
    const float* xr = a.x + (size_t)(n - 1) * a.H;
    float* pv = a.prev + (size_t)a.slots[b] * a.prev_stride;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < a.H; c += gridDim.y * blockDim.x) pv[c] = xr[c];
}

// out: n_mix matrices [T, H] (act_dtype), group_stride elements apart
extern "C" int illm_token_mix(const float* x, int T, int H, int n_mix, const float* mu, float* prev, long long prev_stride, const int* slots,
                              const int* cu_q, const int* token_seq, int B, int single, void* out, int act_dtype, long long group_stride, void* stream) {
    if (T <= 0 || B <= 0) return 0;
    if (H <= 0 || n_mix <= 0 || !x || !mu || !prev || !out || prev_stride < H || group_stride < (long long)T * H || (single && T != B)) return ILLM_ERR_BAD_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    TokenMixArgs a{x, H, n_mix, mu, prev, prev_stride, slots, cu_q, token_seq, group_stride, single};
    const bool vec = !(H & 3) && !(prev_stride & 3) && !(group_stride & 3) && !(((uintptr_t)x | (uintptr_t)mu | (uintptr_t)prev | (uintptr_t)out) & 15);
    const dim3 grid(T, (unsigned)((H + (vec ? 1023 : 255)) / (vec ? 1024 : 256)));
    if (act_dtype == ILLM_BF16 && vec) illm_launch((token_mix_kernel<bf16, 4>), grid, dim3(256), 0, s, a, (bf16*)out);
    else if (act_dtype == ILLM_BF16) illm_launch((token_mix_kernel<bf16, 1>), grid, dim3(256), 0, s, a, (bf16*)out);
    else if (act_dtype == ILLM_F32 && vec) illm_launch((token_mix_kernel<float, 4>), grid, dim3(256), 0, s, a, (float*)out);
    else if (act_dtype == ILLM_F32) illm_launch((token_mix_kernel<float, 1>), grid, dim3(256), 0, s, a, (float*)out);
    else return ILLM_ERR_BAD_ARG;
    if (!single) illm_launch(token_mix_state_kernel, dim3(B, 4), dim3(256), 0, s, a);
    return illm_launch_status();
}

// ---- decay and bonus

struct WkvPrepArgs {
    const float* y;                 // the projections [T, ld]: r, k at r_off, k_off (heads x d), z (rank columns) at z_off
    int T, ld, r_off, k_off, z_off, rank;
    int nh, d;
    const float *w0, *u;            // [nh * d]
    float* w;                       // [T, nh * d]
    float* bonus;                   // [T, nh]
};

// exp(-exp(z)): in (0, 1), 1 where exp(z) rounds away, 0 where it is large
__device__ __forceinline__ float wkv_decay(float z) { return expf(-expf(z)); }

#define WP_TOK 16
#define WP_RK 64

// grid (ceil(T / 16), heads): sixteen tokens of one head; a thread per key channel
template <typename TW>
__global__ void __launch_bounds__(128) wkv_prep_kernel(WkvPrepArgs a, const TW* __restrict__ w2) {
    pdl_grid_sync();
    __shared__ float th[WP_RK][WP_TOK];             // tanh of the inner products, a piece of the rank at a time
    const int t0 = blockIdx.x * WP_TOK, h = blockIdx.y, n = a.T - t0 < WP_TOK ? a.T - t0 : WP_TOK;
    for (int c0 = 0; c0 < a.d; c0 += 128) {
        const int c = c0 + threadIdx.x, ch = h * a.d + c;
        float acc[WP_TOK];
        const float base = c < a.d ? a.w0[ch] : 0.f;
#pragma unroll
        for (int i = 0; i < WP_TOK; i++) acc[i] = 0.f;
        for (int r0 = 0; r0 < a.rank; r0 += WP_RK) {
            const int rn = a.rank - r0 < WP_RK ? a.rank - r0 : WP_RK;
            __syncthreads();
            for (int i = threadIdx.x; i < rn * WP_TOK; i += 128) {
                const int tt = i / rn, r = i - tt * rn;
                th[r][tt] = tt < n ? tanhf(a.y[(size_t)(t0 + tt) * a.ld + a.z_off + r0 + r]) : 0.f;
            }
            __syncthreads();
            if (c < a.d) {
                const TW* row = w2 + (size_t)ch * a.rank + r0;
                for (int r = 0; r < rn; r++) {
                    const float m = to_f32(row[r]);
                    const float4* tv = reinterpret_cast<const float4*>(th[r]);
#pragma unroll
                    for (int i = 0; i < WP_TOK / 4; i++) {
                        const float4 q = tv[i];
                        acc[4 * i] = fmaf(m, q.x, acc[4 * i]);
                        acc[4 * i + 1] = fmaf(m, q.y, acc[4 * i + 1]);
                        acc[4 * i + 2] = fmaf(m, q.z, acc[4 * i + 2]);
                        acc[4 * i + 3] = fmaf(m, q.w, acc[4 * i + 3]);
                    }
                }
            }
        }
        if (c < a.d) {
#pragma unroll
            for (int i = 0; i < WP_TOK; i++)
                if (i < n) a.w[(size_t)(t0 + i) * a.nh * a.d + ch] = wkv_decay(acc[i] + base);
        }
    }
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    for (int tt = warp; tt < n; tt += 4) {
        const float* row = a.y + (size_t)(t0 + tt) * a.ld;
        float s = 0.f;
        for (int c = lane; c < a.d; c += 32) s = fmaf(row[a.r_off + h * a.d + c] * a.u[h * a.d + c], row[a.k_off + h * a.d + c], s);
        s = warp_sum(s);
        if (lane == 0) a.bonus[(size_t)(t0 + tt) * a.nh + h] = s;
    }
}

// ---- the recurrence over a step's tokens, one by one

#define WS_THREADS 128
#define WS_MAX_TILE 16
#define WS_U 4             // tokens whose reductions are interleaved

struct WkvScanArgs {
    const float* y;                 // [T, ld]: r, k, v at their offsets
    int ld, r_off, k_off, v_off;
    int nh, d, dv;
    const float *w, *bonus;         // [T, nh * d], [T, nh]
    float* state;                   // [slots][nh, dv, d], state_stride floats apart
    long long state_stride;
    const int *slots, *cu_q;
    float* out;                     // [T, nh * dv]
    int tile, vec;
};

__device__ __forceinline__ void ws_cp_async16(float* dst, const float* src) {
    const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
}

// A thread's piece of a state [dv][d] at `src`: R = 4 M rows of C columns as pairs of rows; row of pair (m, p): m * 4 LI + 4 g +
// 2 p and the one behind it, so that the LI lanes of a column group touch 16-byte pieces that lie side by side.
template <int C, int M, int LI>
__device__ __forceinline__ void wkv_load_state(f2 (&s)[C][M][2], const float* src, int j, int g, int d, int dv, bool vec) {
#pragma unroll
    for (int c = 0; c < C; c++)
#pragma unroll
        for (int m = 0; m < M; m++) {
            const int i = m * 4 * LI + 4 * g;
            float v[4];
            if (vec && j + c < dv && i < d) {
                const float4 v4 = *reinterpret_cast<const float4*>(src + (size_t)(j + c) * d + i);
                v[0] = v4.x; v[1] = v4.y; v[2] = v4.z; v[3] = v4.w;
            } else {
#pragma unroll
                for (int r = 0; r < 4; r++) v[r] = (j + c < dv && i + r < d) ? src[(size_t)(j + c) * d + i + r] : 0.f;
            }
            s[c][m][0] = f2_pack(v[0], v[1]);
            s[c][m][1] = f2_pack(v[2], v[3]);
        }
}
template <int C, int M, int LI>
__device__ __forceinline__ void wkv_store_state(const f2 (&s)[C][M][2], float* dst, int j, int g, int d, int dv, bool vec) {
#pragma unroll
    for (int c = 0; c < C; c++)
#pragma unroll
        for (int m = 0; m < M; m++) {
            const int i = m * 4 * LI + 4 * g;
            float v[4];
            f2_unpack(s[c][m][0], v[0], v[1]);
            f2_unpack(s[c][m][1], v[2], v[3]);
            if (vec && j + c < dv && i < d) {
                *reinterpret_cast<float4*>(dst + (size_t)(j + c) * d + i) = make_float4(v[0], v[1], v[2], v[3]);
            } else {
#pragma unroll
                for (int r = 0; r < 4; r++)
                    if (j + c < dv && i + r < d) dst[(size_t)(j + c) * d + i + r] = v[r];
            }
        }
}

// The sums of p[u][c] over the LI lanes of a column group, a fixed tree: while a lane holds several columns, each step halves
// them (a lane keeps the lower half if its bit is clear and gets the partner's part of it); with one column left the
// steps are plain.  *first: the first column this lane still holds, *held: how many; false for a lane whose sums another holds too.
template <int U, int C, int LI>
__device__ __forceinline__ bool wkv_lane_sums(float (&p)[U][C], int lane, int* first, int* held) {
    int at = 0, nc = C, plain_bits = 0;
#pragma unroll
    for (int o = LI / 2; o >= 1; o >>= 1) {
        const bool up = (lane & o) != 0;
        if (nc > 1) {
            const int hf = nc / 2;
#pragma unroll
            for (int u = 0; u < U; u++)
#pragma unroll
                for (int c = 0; c < C / 2; c++) {
                    if (c < hf) {
                        const float mine = up ? p[u][c + hf] : p[u][c];
                        const float theirs = up ? p[u][c] : p[u][c + hf];
                        p[u][c] = mine + __shfl_xor_sync(0xffffffffu, theirs, o);
                    }
                }
            if (up) at += hf;
            nc = hf;
        } else {
#pragma unroll
            for (int u = 0; u < U; u++) p[u][0] += __shfl_xor_sync(0xffffffffu, p[u][0], o);
            plain_bits |= o;
        }
    }
    *first = at;
    *held = nc;
    return (lane & plain_bits) == 0;
}

// R rows x C columns of the state per thread, the rows of a column group over LI lanes
template <int R, int C, int LI>
__global__ void __launch_bounds__(WS_THREADS) wkv_scan_kernel(WkvScanArgs a) {
    pdl_grid_sync();
    extern __shared__ __align__(16) float sm[];
    constexpr int M = R / 4;                        // 16-byte pieces of r, k and w per thread
    constexpr int JB = C * (32 / LI) * (WS_THREADS / 32);      // columns per block
    constexpr int DP = R * LI;                      // rows with padding
    constexpr int ROW = 3 * DP + JB + 4;            // floats of one staged token: r, k, w, v, the bonus
    constexpr int V_AT = 3 * DP, B_AT = 3 * DP + JB;
    const int b = blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * JB;
    const int d = a.d, dv = a.dv;
    const int t0 = a.cu_q[b], t1 = a.cu_q[b + 1];
    if (t0 >= t1) return;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int g = lane % LI;
    const int jl = (warp * (32 / LI) + lane / LI) * C;      // first of this thread's columns within the block
    const int jn = dv - j0 < JB ? dv - j0 : JB;     // columns of this block that exist
    float* Sg = a.state + (size_t)a.slots[b] * a.state_stride + (size_t)h * d * dv;       // [dv][d]
    f2 s[C][M][2];
    wkv_load_state<C, M, LI>(s, Sg, j0 + jl, g, d, dv, a.vec);
    // rows beyond d and columns beyond dv stay zero in both buffers
    for (int idx = threadIdx.x; idx < 2 * a.tile * ROW; idx += WS_THREADS) sm[idx] = 0.f;
    __syncthreads();
    auto stage = [&](int buf, int tb) {
        const int n = t1 - tb < a.tile ? t1 - tb : a.tile;
        float* base = sm + buf * a.tile * ROW;
        if (a.vec) {
            const int cq = d >> 2, cv = jn >> 2, per = 3 * cq + cv;
            for (int idx = threadIdx.x; idx < n * per; idx += WS_THREADS) {
                const int tt = idx / per, c = idx - tt * per;
                const float* row = a.y + (size_t)(tb + tt) * a.ld;
                float* dst = base + tt * ROW;
                if (c < cq) ws_cp_async16(dst + 4 * c, row + a.r_off + h * d + 4 * c);
                else if (c < 2 * cq) ws_cp_async16(dst + DP + 4 * (c - cq), row + a.k_off + h * d + 4 * (c - cq));
                else if (c < 3 * cq) ws_cp_async16(dst + 2 * DP + 4 * (c - 2 * cq), a.w + (size_t)(tb + tt) * a.nh * d + h * d + 4 * (c - 2 * cq));
                else ws_cp_async16(dst + V_AT + 4 * (c - 3 * cq), row + a.v_off + h * dv + j0 + 4 * (c - 3 * cq));
            }
        } else {
            const int per = 3 * d + jn;
            for (int idx = threadIdx.x; idx < n * per; idx += WS_THREADS) {
                const int tt = idx / per, c = idx - tt * per;
                const float* row = a.y + (size_t)(tb + tt) * a.ld;
                float* dst = base + tt * ROW;
                if (c < d) dst[c] = row[a.r_off + h * d + c];
                else if (c < 2 * d) dst[DP + c - d] = row[a.k_off + h * d + c - d];
                else if (c < 3 * d) dst[2 * DP + c - 2 * d] = a.w[(size_t)(tb + tt) * a.nh * d + h * d + c - 2 * d];
                else dst[V_AT + c - 3 * d] = row[a.v_off + h * dv + j0 + c - 3 * d];
            }
        }
        for (int tt = threadIdx.x; tt < n; tt += WS_THREADS) base[tt * ROW + B_AT] = a.bonus[(size_t)(tb + tt) * a.nh + h];
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    auto tokens = [&](auto group, const float* rowp, int t) {
        constexpr int U = decltype(group)::value;
        float p[U][C];
#pragma unroll
        for (int u = 0; u < U; u++) {
            const ulonglong2* r4 = reinterpret_cast<const ulonglong2*>(rowp + u * ROW) + g;
            const ulonglong2* k4 = reinterpret_cast<const ulonglong2*>(rowp + u * ROW + DP) + g;
            const ulonglong2* w4 = reinterpret_cast<const ulonglong2*>(rowp + u * ROW + 2 * DP) + g;
            const float* vp = rowp + u * ROW + V_AT + jl;
            f2 v[C], acc[C];
#pragma unroll
            for (int c = 0; c < C; c++) {
                v[c] = f2_pack(vp[c], vp[c]);
                acc[c] = 0;
            }
#pragma unroll
            for (int m = 0; m < M; m++) {
                const ulonglong2 rr = r4[m * LI], kk = k4[m * LI], ww = w4[m * LI];
#pragma unroll
                for (int c = 0; c < C; c++) {
                    acc[c] = f2_fma(s[c][m][0], rr.x, acc[c]);
                    acc[c] = f2_fma(s[c][m][1], rr.y, acc[c]);
                    s[c][m][0] = f2_fma(ww.x, s[c][m][0], f2_mul(kk.x, v[c]));
                    s[c][m][1] = f2_fma(ww.y, s[c][m][1], f2_mul(kk.y, v[c]));
                }
            }
#pragma unroll
            for (int c = 0; c < C; c++) {
                float lo, hi;
                f2_unpack(acc[c], lo, hi);
                p[u][c] = lo + hi;
            }
        }
        int first, held;
        if (wkv_lane_sums<U, C, LI>(p, lane, &first, &held)) {
#pragma unroll
            for (int u = 0; u < U; u++) {
                float* orow = a.out + (size_t)(t + u) * a.nh * dv + (size_t)h * dv + j0 + jl + first;
                const float* vp = rowp + u * ROW + V_AT + jl + first;
                const float bonus = rowp[u * ROW + B_AT];
#pragma unroll
                for (int c = 0; c < C; c++)
                    if (c < held && j0 + jl + first + c < dv) orow[c] = fmaf(bonus, vp[c], p[u][c]);
            }
        }
    };
    stage(0, t0);
    int buf = 0;
    for (int tb = t0; tb < t1; tb += a.tile, buf ^= 1) {
        const int n = t1 - tb < a.tile ? t1 - tb : a.tile;
        if (tb + a.tile < t1) {
            stage(buf ^ 1, tb + a.tile);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const float* base = sm + buf * a.tile * ROW;
        int tt = 0;
        for (; tt + WS_U <= n; tt += WS_U) tokens(std::integral_constant<int, WS_U>(), base + tt * ROW, tb + tt);
        for (; tt < n; tt++) tokens(std::integral_constant<int, 1>(), base + tt * ROW, tb + tt);
        __syncthreads();        // the buffer is filled again by the tile after the next
    }
    wkv_store_state<C, M, LI>(s, Sg, j0 + jl, g, d, dv, a.vec);
}

// head sizes up to 1024 (the rows of a column group over at most 32 lanes), any value size
extern "C" int illm_wkv_supported(int d, int dv) { return d > 0 && d <= 1024 && dv > 0 ? 1 : 0; }

template <int R, int C, int LI>
static void wkv_scan_launch(WkvScanArgs a, int B, cudaStream_t s) {
    constexpr int DP = R * LI, JB = C * (32 / LI) * (WS_THREADS / 32), ROW = 3 * DP + JB + 4;
    int tile = (int)(48 * 1024 / sizeof(float) / (2 * ROW));
    a.tile = tile > WS_MAX_TILE ? WS_MAX_TILE : (tile < 1 ? 1 : tile);
    if (a.tile > WS_U) a.tile -= a.tile % WS_U;
    illm_launch(wkv_scan_kernel<R, C, LI>, dim3(B, a.nh, (a.dv + JB - 1) / JB), dim3(WS_THREADS), (size_t)2 * a.tile * ROW * sizeof(float), s, a);
}

// y: the projections [T, ld] with r, k, v and the decay's inner products z at their offsets; w2 [nh * d, rank] (w2_dtype), w0, u
// float32 [nh * d].  Scratch: w [T, nh * d], bonus [T, nh].  out: float32 [T, nh * dv].
extern "C" int illm_wkv_scan(const float* y, int T, int ld, int r_off, int k_off, int v_off, int z_off, int rank, int nh, int d, int dv, const void* w2,
                             int w2_dtype, const float* w0, const float* u, float* state, long long state_stride, const int* slots, const int* cu_q,
                             float* w, float* bonus, float* out, int B, void* stream) {
    if (B <= 0 || T <= 0) return 0;
    if (nh <= 0 || nh > 65535 || d <= 0 || d > 1024 || dv <= 0 || rank <= 0 || !y || !w2 || !w0 || !u || !state || !w || !bonus || !out ||
        state_stride < (long long)nh * d * dv)
        return ILLM_ERR_BAD_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    WkvPrepArgs p{y, T, ld, r_off, k_off, z_off, rank, nh, d, w0, u, w, bonus};
    const dim3 pgrid((T + WP_TOK - 1) / WP_TOK, nh);
    if (w2_dtype == ILLM_BF16) illm_launch(wkv_prep_kernel<bf16>, pgrid, dim3(128), 0, s, p, (const bf16*)w2);
    else if (w2_dtype == ILLM_F32) illm_launch(wkv_prep_kernel<float>, pgrid, dim3(128), 0, s, p, (const float*)w2);
    else return ILLM_ERR_BAD_ARG;
    WkvScanArgs a{y, ld, r_off, k_off, v_off, nh, d, dv, w, bonus, state, state_stride, slots, cu_q, out, 0, 0};
    a.vec = !((d | dv | ld | r_off | k_off | v_off) & 3) && !((uintptr_t)y & 15) && !((uintptr_t)state & 15) && !((uintptr_t)w & 15) && !(state_stride & 3);
    if (d <= 16) wkv_scan_launch<16, 4, 1>(a, B, s);
    else if (d <= 32) wkv_scan_launch<16, 4, 2>(a, B, s);
    else if (d <= 64) wkv_scan_launch<16, 4, 4>(a, B, s);
    else if (d <= 128) wkv_scan_launch<16, 4, 8>(a, B, s);
    else if (d <= 256) wkv_scan_launch<16, 4, 16>(a, B, s);
    else if (d <= 512) wkv_scan_launch<16, 4, 32>(a, B, s);
    else wkv_scan_launch<32, 2, 32>(a, B, s);
    return illm_launch_status();
}

// ---- sixteen tokens at a time

#define WC_L 16                     // tokens of a chunk
#define WC_CH 128                   // channels that the preparation takes at a time
#define WC_LD (WC_CH + 4)
#define WC_RK 64                    // columns of the low-rank map at a time
#define WC_TLD (WC_RK + 8)

struct WkvChunkPrepArgs {
    float* y;                       // [T, ld]: r and k are replaced by r * P_t and k * Q_t
    int ld, r_off, k_off, z_off, rank;
    int nh, d;
    const bf16* w2;                 // [nh * d, rank]
    const float *w0, *u;
    const int* cu_q;
    float* A;                       // [chunk places, nh, 16, 16]
    float* P;                       // [chunk places, nh, d]
};

// a sequence's chunks have neighbouring places, and no two sequences share one
__device__ __forceinline__ int wc_place(int first_token, int b) { return first_token / WC_L + b; }
extern "C" long long illm_wkv_chunk_places(int T, int B) { return (long long)T / WC_L + B + 1; }

__device__ __forceinline__ void wc_ldsm4(unsigned* r, const void* p) {
    const unsigned addr = (unsigned)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void wc_mma(float* c, const unsigned* a, unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// grid (most chunks of a sequence, heads, sequences)
__global__ void __launch_bounds__(128, 4) wkv_chunk_prep_kernel(WkvChunkPrepArgs a) {
    pdl_grid_sync();
    __shared__ __align__(16) bf16 th[2][WC_L][WC_TLD];             // tanh of the inner products, two bfloat16 terms
    struct Rows { float ws[WC_L][WC_LD], rs[WC_L][WC_LD], ks[WC_L][WC_LD]; };
    union Shared { Rows rows; bf16 w2[WC_CH][WC_TLD]; };           // the outer map's tile is done with before the rows are made
    __shared__ __align__(16) Shared sh;
    float (*ws)[WC_LD] = sh.rows.ws, (*rs)[WC_LD] = sh.rows.rs, (*ks)[WC_LD] = sh.rows.ks;
    __shared__ __align__(16) float us[WC_CH];
    __shared__ float As[WC_L][WC_L];
    const int b = blockIdx.z, h = blockIdx.y, q0 = a.cu_q[b], q1 = a.cu_q[b + 1];
    const int t0 = q0 + blockIdx.x * WC_L, n = q1 - t0 < WC_L ? q1 - t0 : WC_L;
    if (n <= 0) return;
    const size_t place = (size_t)(wc_place(q0, b) + blockIdx.x) * a.nh + h;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, d = a.d;
    for (int i = tid; i < WC_L * WC_L; i += 128) (&As[0][0])[i] = 0.f;
    // A: this thread takes columns s1 and s2 of sixteen rows, of every 128 channels eight (its slice)
    const int slice = tid & 15, s1 = tid >> 4, s2 = WC_L - 1 - s1;
    float av[WC_L + 1];
#pragma unroll
    for (int j = 0; j <= WC_L; j++) av[j] = 0.f;
    for (int c0 = 0; c0 < d; c0 += WC_CH) {
        // this thread's channel of r and k, on its way while the decays are made
        const int ch = c0 + tid;
        float kr[WC_L], rr[WC_L];
        float* yr = a.y + (size_t)t0 * a.ld + a.r_off + h * d + ch;
        float* yk = a.y + (size_t)t0 * a.ld + a.k_off + h * d + ch;
#pragma unroll
        for (int t = 0; t < WC_L; t++) {
            rr[t] = t < n && ch < d ? yr[(size_t)t * a.ld] : 0.f;
            kr[t] = t < n && ch < d ? yk[(size_t)t * a.ld] : 0.f;
        }
        float acc[4][4];
#pragma unroll
        for (int i = 0; i < 4; i++)
#pragma unroll
            for (int k = 0; k < 4; k++) acc[i][k] = 0.f;
        for (int r0 = 0; r0 < a.rank; r0 += WC_RK) {
            __syncthreads();
            if (!(a.rank & 7)) {        // rows of whole 16-byte pieces
                for (int i = tid; i < WC_CH * (WC_RK / 8); i += 128) {
                    const int e = i / (WC_RK / 8), p = i % (WC_RK / 8) * 8;
                    bf16* dst = &sh.w2[e][p];
                    if (c0 + e < d && r0 + p < a.rank)
                        asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((unsigned)__cvta_generic_to_shared(dst)),
                                     "l"(a.w2 + (size_t)(h * d + c0 + e) * a.rank + r0 + p) : "memory");
                    else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
                }
                asm volatile("cp.async.commit_group;" ::: "memory");
            } else {
                for (int i = tid; i < WC_CH * WC_RK; i += 128) {
                    const int e = i / WC_RK, p = i % WC_RK;
                    sh.w2[e][p] = c0 + e < d && r0 + p < a.rank ? a.w2[(size_t)(h * d + c0 + e) * a.rank + r0 + p] : __float2bfloat16_rn(0.f);
                }
            }
            for (int i = tid; i < WC_L * WC_RK; i += 128) {
                const int tt = i / WC_RK, r = i % WC_RK;
                const float v = tt < n && r0 + r < a.rank ? tanhf(a.y[(size_t)(t0 + tt) * a.ld + a.z_off + r0 + r]) : 0.f;
                const bf16 hi = __float2bfloat16_rn(v);
                th[0][tt][r] = hi;
                th[1][tt][r] = __float2bfloat16_rn(v - __bfloat162float(hi));
            }
            asm volatile("cp.async.wait_group 0;" ::: "memory");
            __syncthreads();
            const int steps = ((a.rank - r0 < WC_RK ? a.rank - r0 : WC_RK) + 15) / 16;
            for (int kk = 0; kk < steps; kk++) {
                unsigned hi[4], lo[4];
                wc_ldsm4(hi, &th[0][lane & 15][kk * 16 + (lane >> 4) * 8]);
                wc_ldsm4(lo, &th[1][lane & 15][kk * 16 + (lane >> 4) * 8]);
#pragma unroll
                for (int i = 0; i < 2; i++) {
                    unsigned bb[4];
                    wc_ldsm4(bb, &sh.w2[warp * 32 + i * 16 + (lane & 7) + ((lane >> 4) << 3)][kk * 16 + ((lane >> 3) & 1) * 8]);
                    wc_mma(acc[2 * i], hi, bb[0], bb[1]);
                    wc_mma(acc[2 * i], lo, bb[0], bb[1]);
                    wc_mma(acc[2 * i + 1], hi, bb[2], bb[3]);
                    wc_mma(acc[2 * i + 1], lo, bb[2], bb[3]);
                }
            }
        }
        __syncthreads();        // the rows of the channels before are no longer read
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const int e = (warp * 4 + i) * 8 + (lane & 3) * 2, c = c0 + e;
            const float b0 = c < d ? a.w0[h * d + c] : 0.f, b1 = c + 1 < d ? a.w0[h * d + c + 1] : 0.f;
#pragma unroll
            for (int x = 0; x < 2; x++) {
                const int tt = (lane >> 2) + 8 * x;
                // tokens and channels that are not there leave every product as it is
                ws[tt][e] = tt < n && c < d ? wkv_decay(acc[i][2 * x] + b0) : 1.f;
                ws[tt][e + 1] = tt < n && c + 1 < d ? wkv_decay(acc[i][2 * x + 1] + b1) : 1.f;
            }
        }
        __syncthreads();
        {
            const int c = ch;
            us[tid] = c < d ? a.u[h * d + c] : 0.f;
#pragma unroll
            for (int t = 0; t < WC_L; t++) {
                rs[t][tid] = rr[t];
                ks[t][tid] = kr[t];
            }
            float cum = 1.f;
#pragma unroll
            for (int t = 0; t < WC_L; t++) {
                if (t < n && c < d) yr[(size_t)t * a.ld] = rr[t] * cum;
                cum *= ws[t][tid];
            }
            if (c < d) a.P[place * d + c] = cum;
            float suf = 1.f;
#pragma unroll
            for (int t = WC_L - 1; t >= 0; t--) {
                if (t < n && c < d) yk[(size_t)t * a.ld] = kr[t] * suf;
                suf *= ws[t][tid];
            }
        }
        __syncthreads();
        f2 q[4];
#pragma unroll
        for (int i = 0; i < 4; i++) q[i] = 0;
#pragma unroll
        for (int j = 0; j <= WC_L; j++) {       // rows s1 .. 15 of column s1, then rows s2 .. 15 of column s2
            const bool second = j >= WC_L - s1;
            const int s = second ? s2 : s1, t = second ? s2 + j - (WC_L - s1) : s1 + j;
            const ulonglong2* rp = reinterpret_cast<const ulonglong2*>(&rs[t][slice * 8]);
            const ulonglong2 ra = rp[0], rb = rp[1];
            f2 sum;
            if (t == s) {
                const ulonglong2* kp = reinterpret_cast<const ulonglong2*>(&ks[t][slice * 8]);
                const ulonglong2* up = reinterpret_cast<const ulonglong2*>(&us[slice * 8]);
                const ulonglong2 ka = kp[0], kb = kp[1], ua = up[0], ub = up[1];
                q[0] = ka.x, q[1] = ka.y, q[2] = kb.x, q[3] = kb.y;
                sum = f2_mul(f2_mul(ra.x, ua.x), q[0]);
                sum = f2_fma(f2_mul(ra.y, ua.y), q[1], sum);
                sum = f2_fma(f2_mul(rb.x, ub.x), q[2], sum);
                sum = f2_fma(f2_mul(rb.y, ub.y), q[3], sum);
            } else {
                const ulonglong2* wp = reinterpret_cast<const ulonglong2*>(&ws[t][slice * 8]);
                const ulonglong2 wa = wp[0], wb = wp[1];
                sum = f2_mul(ra.x, q[0]);
                sum = f2_fma(ra.y, q[1], sum);
                sum = f2_fma(rb.x, q[2], sum);
                sum = f2_fma(rb.y, q[3], sum);
                q[0] = f2_mul(q[0], wa.x), q[1] = f2_mul(q[1], wa.y), q[2] = f2_mul(q[2], wb.x), q[3] = f2_mul(q[3], wb.y);
            }
            float lo, hi;
            f2_unpack(sum, lo, hi);
            av[j] += lo + hi;
        }
    }
#pragma unroll
    for (int j = 0; j <= WC_L; j++) {
        float v = av[j];
#pragma unroll
        for (int o = 8; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
        const bool second = j >= WC_L - s1;
        if (slice == 0) As[second ? s2 + j - (WC_L - s1) : s1 + j][second ? s2 : s1] = v;
    }
    __syncthreads();
    for (int i = tid; i < WC_L * WC_L; i += 128) a.A[place * WC_L * WC_L + i] = (&As[0][0])[i];
}

struct WkvChunkArgs {
    const float* y;                 // [T, ld] as the preparation left it, v untouched
    int ld, r_off, k_off, v_off;
    int nh, d, dv;
    const float *A, *P;
    float* state;
    long long state_stride;
    const int *slots, *cu_q;
    float* out;                     // [T, nh * dv]
    int segments;
    float* seg_state;               // [B, segments, nh, dv, d]; the last place keeps the state that came in
    float* seg_decay;               // [B, segments, nh, d]
};

template <int R, int C, int LI, int PASS>
__global__ void __launch_bounds__(128) wkv_chunk_kernel(WkvChunkArgs a) {
    pdl_grid_sync();
    extern __shared__ __align__(16) float sm[];
    constexpr int M = R / 4, DP = R * LI, JB = C * (32 / LI) * 4;
    constexpr int U = C >= 8 ? 2 : 4;               // tokens whose sums are interleaved
    constexpr int R_AT = 0, K_AT = PASS ? WC_L * DP : 0, V_AT = K_AT + WC_L * DP, P_AT = V_AT + WC_L * JB, A_AT = P_AT + DP;
    constexpr int TILE = A_AT + (PASS ? WC_L * WC_L : 0);
    constexpr int NP = LI >= 8 ? 1 : 8 / LI;        // pairs of a chunk's tokens per lane in the sum over A
    const int S = a.segments;
    const int b = blockIdx.x / S, seg = blockIdx.x % S, h = blockIdx.y, j0 = blockIdx.z * JB, d = a.d, dv = a.dv;
    const int q0 = a.cu_q[b], q1 = a.cu_q[b + 1], chunks = (q1 - q0 + WC_L - 1) / WC_L, per = (chunks + S - 1) / S;
    const int first_chunk = seg * per, end_chunk = first_chunk + per < chunks ? first_chunk + per : chunks;
    if (first_chunk >= end_chunk) return;           // a short sequence fills fewer segments
    const bool last = end_chunk == chunks;
    if (PASS == 0 && last) return;                  // nobody starts from the last segment's state
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane % LI;
    const int jl = (warp * (32 / LI) + lane / LI) * C;
    const int jn = dv - j0 < JB ? dv - j0 : JB;
    float* Sg = a.state + (size_t)a.slots[b] * a.state_stride + (size_t)h * d * dv;       // [dv][d]
    float* seg_base = a.seg_state + ((size_t)b * S * a.nh + h) * (size_t)d * dv;          // + segment * nh * d * dv
    const size_t seg_stride = (size_t)a.nh * d * dv;
    float* dec_base = a.seg_decay + ((size_t)b * S * a.nh + h) * (size_t)d;
    const size_t dec_stride = (size_t)a.nh * d;
    const size_t place0 = (size_t)wc_place(q0, b);
    for (int idx = threadIdx.x; idx < 2 * TILE; idx += 128) sm[idx] = 0.f;          // rows beyond d, columns beyond dv, tokens that are not there
    __syncthreads();
    auto stage = [&](int buf, int chunk) {
        const int t0 = q0 + chunk * WC_L, n = q1 - t0 < WC_L ? q1 - t0 : WC_L;
        float* base = sm + buf * TILE;
        const int cq = d >> 2, cv = jn >> 2;
        const float* row0 = a.y + (size_t)t0 * a.ld;
        for (int tt = warp; tt < n; tt += 4) {
            const float* row = row0 + (size_t)tt * a.ld;
            for (int c = lane; c < cq; c += 32) {
                if (PASS == 1) ws_cp_async16(base + R_AT + tt * DP + 4 * c, row + a.r_off + h * d + 4 * c);
                ws_cp_async16(base + K_AT + tt * DP + 4 * c, row + a.k_off + h * d + 4 * c);
            }
            for (int c = lane; c < cv; c += 32) ws_cp_async16(base + V_AT + tt * JB + 4 * c, row + a.v_off + h * dv + j0 + 4 * c);
        }
        const size_t place = (place0 + chunk) * a.nh + h;
        for (int c = threadIdx.x; c < cq; c += 128) ws_cp_async16(base + P_AT + 4 * c, a.P + place * d + 4 * c);
        if (PASS == 1 && threadIdx.x < WC_L * WC_L / 4) ws_cp_async16(base + A_AT + 4 * threadIdx.x, a.A + place * WC_L * WC_L + 4 * threadIdx.x);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(0, first_chunk);
    f2 s[C][M][2], cum[M][2];
    if (PASS == 0) {
#pragma unroll
        for (int m = 0; m < M; m++) cum[m][0] = cum[m][1] = f2_pack(1.f, 1.f);
        if (seg == 0) {
            // what came in is kept for pass 1, whose last segment renews the state while its first may not have begun
            wkv_load_state<C, M, LI>(s, Sg, j0 + jl, g, d, dv, true);
            wkv_store_state<C, M, LI>(s, seg_base + (size_t)(S - 1) * seg_stride, j0 + jl, g, d, dv, true);
        } else {
#pragma unroll
            for (int c = 0; c < C; c++)
#pragma unroll
                for (int m = 0; m < M; m++) s[c][m][0] = s[c][m][1] = 0;
        }
    } else if (seg == 0) {
        wkv_load_state<C, M, LI>(s, last ? Sg : seg_base + (size_t)(S - 1) * seg_stride, j0 + jl, g, d, dv, true);
    } else {
        wkv_load_state<C, M, LI>(s, seg_base + (seg - 1) * seg_stride, j0 + jl, g, d, dv, true);
    }
    int buf = 0;
    for (int chunk = first_chunk; chunk < end_chunk; chunk++, buf ^= 1) {
        const int t0 = q0 + chunk * WC_L, n = q1 - t0 < WC_L ? q1 - t0 : WC_L;
        if (chunk + 1 < end_chunk) {
            stage(buf ^ 1, chunk + 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const float* base = sm + buf * TILE;
        if (PASS == 1) {
            // a lane's share of the sum over the chunk's own tokens: pairs (2 i, 2 i + 1), i = g, g + LI, ..
            f2 vp[NP][C];
#pragma unroll
            for (int i = 0; i < NP; i++)
#pragma unroll
                for (int c = 0; c < C; c++) {
                    const int s0 = 2 * ((g & 7) + i * LI);
                    vp[i][c] = LI <= 8 || g < 8 ? f2_pack(base[V_AT + s0 * JB + jl + c], base[V_AT + (s0 + 1) * JB + jl + c]) : 0;
                }
            for (int tt = 0; tt < n; tt += U) {
                float p[U][C];
#pragma unroll
                for (int u = 0; u < U; u++) {
                    const ulonglong2* r4 = reinterpret_cast<const ulonglong2*>(base + R_AT + (tt + u) * DP) + g;
                    f2 acc[C];
#pragma unroll
                    for (int i = 0; i < NP; i++) {
                        const f2 av = *reinterpret_cast<const f2*>(base + A_AT + (tt + u) * WC_L + 2 * ((g & 7) + i * LI));
#pragma unroll
                        for (int c = 0; c < C; c++) acc[c] = i == 0 ? f2_mul(av, vp[i][c]) : f2_fma(av, vp[i][c], acc[c]);
                    }
#pragma unroll
                    for (int m = 0; m < M; m++) {
                        const ulonglong2 rr = r4[m * LI];
#pragma unroll
                        for (int c = 0; c < C; c++) {
                            acc[c] = f2_fma(s[c][m][0], rr.x, acc[c]);
                            acc[c] = f2_fma(s[c][m][1], rr.y, acc[c]);
                        }
                    }
#pragma unroll
                    for (int c = 0; c < C; c++) {
                        float lo, hi;
                        f2_unpack(acc[c], lo, hi);
                        p[u][c] = lo + hi;
                    }
                }
                int first, held;
                if (wkv_lane_sums<U, C, LI>(p, lane, &first, &held)) {
#pragma unroll
                    for (int u = 0; u < U; u++) {
                        float* orow = a.out + (size_t)(t0 + tt + u) * a.nh * dv + (size_t)h * dv + j0 + jl + first;
#pragma unroll
                        for (int c = 0; c < C; c++)
                            if (c < held && tt + u < n && j0 + jl + first + c < dv) orow[c] = p[u][c];
                    }
                }
            }
        }
        const ulonglong2* p4 = reinterpret_cast<const ulonglong2*>(base + P_AT) + g;
#pragma unroll
        for (int m = 0; m < M; m++) {
            const ulonglong2 pp = p4[m * LI];
#pragma unroll
            for (int c = 0; c < C; c++) {
                s[c][m][0] = f2_mul(s[c][m][0], pp.x);
                s[c][m][1] = f2_mul(s[c][m][1], pp.y);
            }
            if (PASS == 0) {
                cum[m][0] = f2_mul(cum[m][0], pp.x);
                cum[m][1] = f2_mul(cum[m][1], pp.y);
            }
        }
#pragma unroll 2
        for (int tt = 0; tt < n; tt++) {
            const ulonglong2* k4 = reinterpret_cast<const ulonglong2*>(base + K_AT + tt * DP) + g;
            const float* vr = base + V_AT + tt * JB + jl;
            f2 v[C];
#pragma unroll
            for (int c = 0; c < C; c++) v[c] = f2_pack(vr[c], vr[c]);
#pragma unroll
            for (int m = 0; m < M; m++) {
                const ulonglong2 kk = k4[m * LI];
#pragma unroll
                for (int c = 0; c < C; c++) {
                    s[c][m][0] = f2_fma(kk.x, v[c], s[c][m][0]);
                    s[c][m][1] = f2_fma(kk.y, v[c], s[c][m][1]);
                }
            }
        }
        __syncthreads();        // the buffer is filled again by the chunk after the next
    }
    if (PASS == 0) {
        wkv_store_state<C, M, LI>(s, seg_base + seg * seg_stride, j0 + jl, g, d, dv, true);
        if (blockIdx.z == 0 && warp == 0 && lane < LI) {
            float* dst = dec_base + seg * dec_stride;
#pragma unroll
            for (int m = 0; m < M; m++) {
                const int i = m * 4 * LI + 4 * g;
                float v[4];
                f2_unpack(cum[m][0], v[0], v[1]);
                f2_unpack(cum[m][1], v[2], v[3]);
                if (i < d) *reinterpret_cast<float4*>(dst + i) = make_float4(v[0], v[1], v[2], v[3]);
            }
        }
    } else if (last) {
        wkv_store_state<C, M, LI>(s, Sg, j0 + jl, g, d, dv, true);
    }
}

// Between the passes: the state behind segment r from those of the segments by themselves, S_r <- diag(D_r) S_(r-1) + S_r, r from
// 1 to the last segment but one.  A thread per four rows of a column.  grid (pieces, heads, sequences)
__global__ void __launch_bounds__(256) wkv_fold_kernel(WkvChunkArgs a) {
    pdl_grid_sync();
    const int S = a.segments, b = blockIdx.z, h = blockIdx.y, d = a.d;
    const int n = a.cu_q[b + 1] - a.cu_q[b], chunks = (n + WC_L - 1) / WC_L, per = (chunks + S - 1) / S;
    const int used = per > 0 ? (chunks + per - 1) / per : 0;
    const int i = (blockIdx.x * 256 + threadIdx.x) * 4;
    if (i >= d * a.dv) return;
    float* st = a.seg_state + ((size_t)b * S * a.nh + h) * (size_t)d * a.dv + i;
    const float* dec = a.seg_decay + ((size_t)b * S * a.nh + h) * (size_t)d + i % d;
    const size_t st_stride = (size_t)a.nh * d * a.dv, dec_stride = (size_t)a.nh * d;
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int r0 = 0; r0 < used - 1; r0 += 4) {
        float4 v[4], f[4];
#pragma unroll
        for (int k = 0; k < 4; k++)
            if (r0 + k < used - 1) {
                v[k] = *reinterpret_cast<const float4*>(st + (r0 + k) * st_stride);
                f[k] = *reinterpret_cast<const float4*>(dec + (r0 + k) * dec_stride);
            }
#pragma unroll
        for (int k = 0; k < 4; k++)
            if (r0 + k < used - 1) {
                acc.x = fmaf(f[k].x, acc.x, v[k].x), acc.y = fmaf(f[k].y, acc.y, v[k].y), acc.z = fmaf(f[k].z, acc.z, v[k].z), acc.w = fmaf(f[k].w, acc.w, v[k].w);
                *reinterpret_cast<float4*>(st + (r0 + k) * st_stride) = acc;
            }
    }
}

template <int R, int C, int LI>
static int wkv_chunk_launch(const WkvChunkArgs& a, int B, cudaStream_t s) {
    constexpr int DP = R * LI, JB = C * (32 / LI) * 4;
    constexpr size_t smem0 = 2 * sizeof(float) * (WC_L * DP + WC_L * JB + DP), smem1 = smem0 + 2 * sizeof(float) * (WC_L * DP + WC_L * WC_L);
    static bool raised = false;
    if (!raised) {
        cudaError_t e = cudaFuncSetAttribute(wkv_chunk_kernel<R, C, LI, 0>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem0);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(wkv_chunk_kernel<R, C, LI, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem1);
        if (e != cudaSuccess) return (int)e;
        raised = true;
    }
    const dim3 grid(B * a.segments, a.nh, (a.dv + JB - 1) / JB);
    if (a.segments > 1) {
        illm_launch(wkv_chunk_kernel<R, C, LI, 0>, grid, dim3(128), smem0, s, a);
        if (a.segments > 2) illm_launch(wkv_fold_kernel, dim3((a.d * a.dv / 4 + 255) / 256, a.nh, B), dim3(256), 0, s, a);
    }
    illm_launch(wkv_chunk_kernel<R, C, LI, 1>, grid, dim3(128), smem1, s, a);
    return illm_launch_status();
}

// rows of whole 16-byte pieces and up to 512 key channels; ld and the offsets are multiples of four too
extern "C" int illm_wkv_chunk_supported(int d, int dv, int ld, int r_off, int k_off, int v_off) {
    return d > 0 && d <= 512 && dv > 0 && !((d | dv | ld | r_off | k_off | v_off) & 3) ? 1 : 0;
}

// The prompts' form: as illm_wkv_scan with w2 in bfloat16; y's r and k columns are scratch afterwards.  A [places, nh, 16, 16] and
// P [places, nh, d] are scratch (places = illm_wkv_chunk_places), with segments > 1 also seg_state [B, segments, nh, dv, d] and
// seg_decay [B, segments, nh, d].  max_q: the most tokens of a sequence.
extern "C" int illm_wkv_chunks(float* y, int T, int ld, int r_off, int k_off, int v_off, int z_off, int rank, int nh, int d, int dv, const void* w2,
                               const float* w0, const float* u, float* state, long long state_stride, const int* slots, const int* cu_q, float* A, float* P,
                               float* out, int B, int max_q, int segments, float* seg_state, float* seg_decay, void* stream) {
    if (B <= 0 || T <= 0) return 0;
    if (segments < 1 || (segments > 1 && (!seg_state || !seg_decay)) || (long long)B * segments > 0x7fffffff || B > 65535 || max_q <= 0) return ILLM_ERR_BAD_ARG;
    if (nh <= 0 || nh > 65535 || rank <= 0 || !y || !w2 || !w0 || !u || !state || !A || !P || !out || state_stride < (long long)nh * d * dv ||
        !illm_wkv_chunk_supported(d, dv, ld, r_off, k_off, v_off) || (state_stride & 3) ||
        (((uintptr_t)y | (uintptr_t)state | (uintptr_t)A | (uintptr_t)P | (uintptr_t)seg_state | (uintptr_t)seg_decay) & 15) || ((uintptr_t)w2 & 15))
        return ILLM_ERR_BAD_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    WkvChunkPrepArgs p{y, ld, r_off, k_off, z_off, rank, nh, d, (const bf16*)w2, w0, u, cu_q, A, P};
    illm_launch(wkv_chunk_prep_kernel, dim3((max_q + WC_L - 1) / WC_L, nh, B), dim3(128), 0, s, p);
    WkvChunkArgs a{y, ld, r_off, k_off, v_off, nh, d, dv, A, P, state, state_stride, slots, cu_q, out, segments, seg_state, seg_decay};
    if (d <= 16) return wkv_chunk_launch<16, 4, 1>(a, B, s);
    if (d <= 32) return wkv_chunk_launch<16, 4, 2>(a, B, s);
    if (d <= 64) return wkv_chunk_launch<16, 4, 4>(a, B, s);
    if (d <= 128) return wkv_chunk_launch<16, 8, 8>(a, B, s);
    if (d <= 256) return wkv_chunk_launch<16, 8, 16>(a, B, s);
    return wkv_chunk_launch<16, 8, 32>(a, B, s);
}

// ---- one token per sequence

struct WkvStepArgs {
    const float* y;                 // the projections [T, ld], finished or as `splits` slices `stride` floats apart
    int splits;
    long long stride;
    int ld, r_off, k_off, v_off, g_off, z_off, rank;
    int nh, d, dv;
    const bf16* w2;                 // [nh * d, rank]
    const float *w0, *u;
    float* state;
    long long state_stride;
    const int* slots;
    const float* norm_w;            // [nh * dv]
    float eps;
};

// grid (tokens, heads), 256 threads: token t is the only one of sequence t.  A column of the state lies over LI lanes, NV pieces
// of four rows each; a warp has CB columns per lane group on their way at a time.
template <int LI, int NV, int CB>
__global__ void __launch_bounds__(256) wkv_step_kernel(WkvStepArgs a, bf16* __restrict__ out) {
    pdl_grid_sync();
    extern __shared__ __align__(16) float sm[];
    __shared__ float scratch[32];
    constexpr int GW = 32 / LI;                     // column groups of a warp
    const int t = blockIdx.x, h = blockIdx.y, d = a.d, dv = a.dv, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane % LI;
    float *r = sm, *k = r + d, *w = k + d, *v = w + d, *gt = v + dv, *o = gt + dv, *th = o + dv;
    float* Sg = a.state + (size_t)a.slots[t] * a.state_stride + (size_t)h * d * dv;
    float4 s[CB][NV];
    auto column = [&](int batch, int c) { return ((batch * CB + c) * 8 + warp) * GW + lane / LI; };
    auto load = [&](int batch) {
#pragma unroll
        for (int c = 0; c < CB; c++) {
            const int j = column(batch, c);
#pragma unroll
            for (int m = 0; m < NV; m++) {
                const int i = 4 * (g + m * LI);
                s[c][m] = j < dv && i < d ? *reinterpret_cast<const float4*>(Sg + (size_t)j * d + i) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
        }
    };
    load(0);
    const float* row = a.y + (size_t)t * a.ld;
    auto projected = [&](int col) {                 // the slices in ascending order, their loads in flight together
        float x = row[col];
        int sl = 1;
        for (; sl + 4 <= a.splits; sl += 4) {
            float f[4];
#pragma unroll
            for (int i = 0; i < 4; i++) f[i] = row[(size_t)(sl + i) * a.stride + col];
#pragma unroll
            for (int i = 0; i < 4; i++) x += f[i];
        }
        for (; sl < a.splits; sl++) x += row[(size_t)sl * a.stride + col];
        return x;
    };
    for (int i = tid; i < 2 * d + 2 * dv + a.rank; i += 256) {
        if (i < d) r[i] = projected(a.r_off + h * d + i);
        else if (i < 2 * d) k[i - d] = projected(a.k_off + h * d + i - d);
        else if (i < 2 * d + dv) v[i - 2 * d] = projected(a.v_off + h * dv + i - 2 * d);
        else if (i < 2 * d + 2 * dv) gt[i - 2 * d - dv] = projected(a.g_off + h * dv + i - 2 * d - dv);
        else th[i - 2 * d - 2 * dv] = tanhf(projected(a.z_off + i - 2 * d - 2 * dv));
    }
    __syncthreads();
    float bonus = 0.f;
    for (int c = tid; c < d; c += 256) bonus = fmaf(r[c] * a.u[h * d + c], k[c], bonus);
    bonus = block_sum(bonus, scratch);
    // two lanes per channel, each half of the low-rank map's columns
    const int half = (a.rank + 15) / 16 * 8;
    for (int i = tid; i < (2 * d + 31) / 32 * 32; i += 256) {
        const int c = i >> 1, r0 = (i & 1) * half, r1 = r0 + half < a.rank ? r0 + half : a.rank;
        float acc = 0.f;
        if (c < d) {
            const bf16* wr = a.w2 + (size_t)(h * d + c) * a.rank;
            if (!(a.rank & 7)) {
                for (int q = r0; q < r1; q += 8) {
                    float f[8];
                    load8(wr + q, f);
#pragma unroll
                    for (int e = 0; e < 8; e++) acc = fmaf(f[e], th[q + e], acc);
                }
            } else {
                for (int q = r0; q < r1; q++) acc = fmaf(to_f32(wr[q]), th[q], acc);
            }
        }
        acc += __shfl_xor_sync(0xffffffffu, acc, 1);
        if (c < d && !(i & 1)) w[c] = wkv_decay(acc + a.w0[h * d + c]);
    }
    __syncthreads();
    float4 r4[NV], k4[NV], w4[NV];
#pragma unroll
    for (int m = 0; m < NV; m++) {
        const int i = 4 * (g + m * LI);
        const bool ok = i < d;
        r4[m] = ok ? *reinterpret_cast<const float4*>(r + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        k4[m] = ok ? *reinterpret_cast<const float4*>(k + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        w4[m] = ok ? *reinterpret_cast<const float4*>(w + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const int batches = (dv + 8 * GW * CB - 1) / (8 * GW * CB);
    for (int batch = 0; batch < batches; batch++) {
        if (batch) load(batch);
        float p[1][CB];
#pragma unroll
        for (int c = 0; c < CB; c++) {
            const int j = column(batch, c);
            const float vj = j < dv ? v[j] : 0.f;
            float x = 0.f;
#pragma unroll
            for (int m = 0; m < NV; m++) {
                float4 q = s[c][m];
                x = fmaf(q.x, r4[m].x, x), x = fmaf(q.y, r4[m].y, x), x = fmaf(q.z, r4[m].z, x), x = fmaf(q.w, r4[m].w, x);
                q.x = fmaf(w4[m].x, q.x, k4[m].x * vj);
                q.y = fmaf(w4[m].y, q.y, k4[m].y * vj);
                q.z = fmaf(w4[m].z, q.z, k4[m].z * vj);
                q.w = fmaf(w4[m].w, q.w, k4[m].w * vj);
                const int i = 4 * (g + m * LI);
                if (j < dv && i < d) *reinterpret_cast<float4*>(Sg + (size_t)j * d + i) = q;
            }
            p[0][c] = x;
        }
        int first, held;
        if (wkv_lane_sums<1, CB, LI>(p, lane, &first, &held)) {
#pragma unroll
            for (int c = 0; c < CB; c++) {
                const int j = column(batch, first + c);
                if (c < held && j < dv) o[j] = fmaf(bonus, v[j], p[0][c]);
            }
        }
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = tid; c < dv; c += 256) ss = fmaf(o[c], o[c], ss);
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)dv + a.eps);
    bf16* orow = out + (size_t)t * a.nh * dv + (size_t)h * dv;
    for (int c = tid; c < dv; c += 256) orow[c] = __float2bfloat16_rn(((o[c] * inv) * a.norm_w[h * dv + c]) * (gt[c] / (1.0f + expf(-gt[c]))));
}

extern "C" int illm_wkv_step_supported(int d, int dv) { return d > 0 && d <= 512 && !(d & 3) && dv > 0 && dv <= 1024 && !(dv & 3) ? 1 : 0; }

// One token per sequence (T = B tokens in the order of the sequences), bfloat16 mode: y [T, ld] float32 with r, k, v, the gate's and
// the decay's inner projections, finished (splits 1) or as slices `stride` floats apart; w2 [nh * d, rank] bfloat16.  out: bfloat16
// [T, nh * dv] = o / rms(o) per head * norm_w * silu(gate).
extern "C" int illm_wkv_step(const float* y, int splits, long long stride, int T, int ld, int r_off, int k_off, int v_off, int g_off, int z_off, int rank,
                             int nh, int d, int dv, const void* w2, const float* w0, const float* u, float* state, long long state_stride,
                             const int* slots, const float* norm_w, float eps, void* out, void* stream) {
    if (T <= 0) return 0;
    if (splits < 1 || nh <= 0 || nh > 65535 || rank <= 0 || rank > 4096 || !y || !w2 || !w0 || !u || !state || !norm_w || !out ||
        !illm_wkv_step_supported(d, dv) || state_stride < (long long)nh * d * dv || (state_stride & 3) || ((uintptr_t)state & 15) || ((uintptr_t)w2 & 15))
        return ILLM_ERR_BAD_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    WkvStepArgs a{y, splits, stride, ld, r_off, k_off, v_off, g_off, z_off, rank, nh, d, dv, (const bf16*)w2, w0, u, state, state_stride, slots, norm_w, eps};
    const size_t smem = (size_t)(3 * d + 3 * dv + rank) * sizeof(float);
    const dim3 grid(T, nh);
    if (d <= 16) illm_launch((wkv_step_kernel<4, 1, 4>), grid, dim3(256), smem, s, a, (bf16*)out);
    else if (d <= 32) illm_launch((wkv_step_kernel<8, 1, 4>), grid, dim3(256), smem, s, a, (bf16*)out);
    else if (d <= 64) illm_launch((wkv_step_kernel<16, 1, 8>), grid, dim3(256), smem, s, a, (bf16*)out);
    else if (d <= 128) illm_launch((wkv_step_kernel<32, 1, 16>), grid, dim3(256), smem, s, a, (bf16*)out);
    else if (d <= 256) illm_launch((wkv_step_kernel<32, 2, 8>), grid, dim3(256), smem, s, a, (bf16*)out);
    else illm_launch((wkv_step_kernel<32, 4, 4>), grid, dim3(256), smem, s, a, (bf16*)out);
    return illm_launch_status();
}
