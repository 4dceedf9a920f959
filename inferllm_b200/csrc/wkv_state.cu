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
// wkv_scan_kernel        the recurrence for steps of any length
// wkv_step_kernel        the recurrence, the decay, the bonus, the per-head unit norm and the gate for one token per sequence
//                        in one kernel, reading the projections as unreduced K slices (the bfloat16 mode's decoding)
//
// wkv_scan_kernel: the columns of S never meet, so a block owns (sequence, head, 64 columns or what the head size leaves) and a
// thread keeps 16 rows of four columns in registers for the whole step, the rows of a column group over LI neighbouring
// lanes, as the scan with one decay per head does (decay_state.cu); here r, k and w of a token are three staged rows, and two
// rows of the state share one instruction (fma.rn.f32x2).  A long prompt of few sequences may be cut into segments that run
// side by side: pass 0 runs each from zero (the first from the sequence's state) and leaves its final state and the product of
// its decays per channel; pass 1 folds the earlier segments' states into the state at the segment's start and adds what that
// state gives its tokens, o_t += S_in^T (r_t * product of the segment's decays before t).  Products of decays are never
// divided by one another.  The sums then have another order than token by token, so the float32 mode never asks for segments.
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

// ---- the recurrence over a step's tokens

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
    int segments;
    float* seg_state;               // [B, segments, nh, dv, d]
    float* seg_decay;               // [B, segments, nh, d]
};

__device__ __forceinline__ void ws_cp_async16(float* dst, const float* src) {
    const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
}

// R rows x C columns of the state per thread, the rows of a column group over LI lanes
template <int R, int C, int LI, int PASS>
__global__ void __launch_bounds__(WS_THREADS) wkv_scan_kernel(WkvScanArgs a) {
    pdl_grid_sync();
    extern __shared__ __align__(16) float sm[];
    constexpr int M = R / 4;                        // 16-byte pieces of r, k and w per thread
    constexpr int JB = C * (32 / LI) * (WS_THREADS / 32);      // columns per block
    constexpr int DP = R * LI;                      // rows with padding
    constexpr int ROW = 3 * DP + JB + 4;            // floats of one staged token: r, k, w, v, the bonus
    constexpr int V_AT = 3 * DP, B_AT = 3 * DP + JB;
    const int P = a.segments;
    const int b = blockIdx.x / P, seg = blockIdx.x % P, h = blockIdx.y, j0 = blockIdx.z * JB;
    const int d = a.d, dv = a.dv;
    const int q0 = a.cu_q[b], q1 = a.cu_q[b + 1];
    const int seg_len = P > 1 ? (((q1 - q0 + P - 1) / P + 15) & ~15) : q1 - q0;      // whole tiles
    const int t0 = q0 + seg * seg_len, t1 = t0 + seg_len < q1 ? t0 + seg_len : q1;
    if (t0 >= t1) return;                                                           // a short sequence fills fewer segments
    const bool last_seg = t1 == q1;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int g = lane % LI;
    const int jl = (warp * (32 / LI) + lane / LI) * C;      // first of this thread's columns within the block
    const int jn = dv - j0 < JB ? dv - j0 : JB;     // columns of this block that exist
    float* Sg = a.state + (size_t)a.slots[b] * a.state_stride + (size_t)h * d * dv;       // [dv][d]
    // row of register pair (m, p): m * 4 LI + 4 g + 2 p and the one behind it
    f2 s[C][M][2];
    f2 cum[M][2];                   // pass 0: the product of the segment's decays so far; pass 1: of those before the token at hand
    const bool keep_cum = PASS == 1 || P > 1;
    // s = (accumulate ? s * mul : 0) + src, per element; mul: the rows' factors or nullptr (1)
    auto load_state = [&](const float* src, const float* mul, bool accumulate) {
#pragma unroll
        for (int c = 0; c < C; c++) {
            const int j = j0 + jl + c;
#pragma unroll
            for (int m = 0; m < M; m++) {
                const int i = m * 4 * LI + 4 * g;
                float v[4], f[4];
                if (a.vec && j < dv && i < d) {
                    const float4 v4 = *reinterpret_cast<const float4*>(src + (size_t)j * d + i);
                    v[0] = v4.x; v[1] = v4.y; v[2] = v4.z; v[3] = v4.w;
                } else {
#pragma unroll
                    for (int r = 0; r < 4; r++) v[r] = (j < dv && i + r < d) ? src[(size_t)j * d + i + r] : 0.f;
                }
                if (accumulate) {
#pragma unroll
                    for (int r = 0; r < 4; r++) f[r] = i + r < d ? mul[i + r] : 0.f;
                    s[c][m][0] = f2_fma(s[c][m][0], f2_pack(f[0], f[1]), f2_pack(v[0], v[1]));
                    s[c][m][1] = f2_fma(s[c][m][1], f2_pack(f[2], f[3]), f2_pack(v[2], v[3]));
                } else {
                    s[c][m][0] = f2_pack(v[0], v[1]);
                    s[c][m][1] = f2_pack(v[2], v[3]);
                }
            }
        }
    };
    auto store_state = [&](float* dst) {
#pragma unroll
        for (int c = 0; c < C; c++) {
            const int j = j0 + jl + c;
#pragma unroll
            for (int m = 0; m < M; m++) {
                const int i = m * 4 * LI + 4 * g;
                float v[4];
                f2_unpack(s[c][m][0], v[0], v[1]);
                f2_unpack(s[c][m][1], v[2], v[3]);
                if (a.vec && j < dv && i < d) {
                    *reinterpret_cast<float4*>(dst + (size_t)j * d + i) = make_float4(v[0], v[1], v[2], v[3]);
                } else {
#pragma unroll
                    for (int r = 0; r < 4; r++)
                        if (j < dv && i + r < d) dst[(size_t)j * d + i + r] = v[r];
                }
            }
        }
    };
    float* seg_base = a.seg_state + ((size_t)b * P * a.nh + h) * (size_t)d * dv;      // + seg * nh * d * dv per segment
    const size_t seg_stride = (size_t)a.nh * d * dv;
    float* dec_base = a.seg_decay + ((size_t)b * P * a.nh + h) * (size_t)d;           // + seg * nh * d per segment
    const size_t dec_stride = (size_t)a.nh * d;
#pragma unroll
    for (int m = 0; m < M; m++) cum[m][0] = cum[m][1] = f2_pack(1.f, 1.f);
    if (PASS == 0) {
        if (seg == 0) {
            load_state(Sg, nullptr, false);
        } else {
#pragma unroll
            for (int c = 0; c < C; c++)
#pragma unroll
                for (int m = 0; m < M; m++) s[c][m][0] = s[c][m][1] = f2_pack(0.f, 0.f);
        }
    } else {
        if (seg == 0) {             // nothing to correct; a sequence of one segment still has to get its state
            if (last_seg) {
                load_state(seg_base, nullptr, false);
                store_state(Sg);
            }
            return;
        }
        load_state(seg_base, nullptr, false);
        for (int r = 1; r < seg; r++) load_state(seg_base + r * seg_stride, dec_base + r * dec_stride, true);
    }
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
                if (PASS == 0) v[c] = f2_pack(vp[c], vp[c]);
                acc[c] = f2_pack(0.f, 0.f);
            }
#pragma unroll
            for (int m = 0; m < M; m++) {
                ulonglong2 rr = r4[m * LI];
                const ulonglong2 ww = w4[m * LI];
                if (PASS == 1) {
                    rr.x = f2_mul(rr.x, cum[m][0]);
                    rr.y = f2_mul(rr.y, cum[m][1]);
                }
                if (PASS == 0) {
                    const ulonglong2 kk = k4[m * LI];
#pragma unroll
                    for (int c = 0; c < C; c++) {
                        acc[c] = f2_fma(s[c][m][0], rr.x, acc[c]);
                        acc[c] = f2_fma(s[c][m][1], rr.y, acc[c]);
                        s[c][m][0] = f2_fma(ww.x, s[c][m][0], f2_mul(kk.x, v[c]));
                        s[c][m][1] = f2_fma(ww.y, s[c][m][1], f2_mul(kk.y, v[c]));
                    }
                } else {
#pragma unroll
                    for (int c = 0; c < C; c++) {
                        acc[c] = f2_fma(s[c][m][0], rr.x, acc[c]);
                        acc[c] = f2_fma(s[c][m][1], rr.y, acc[c]);
                    }
                }
                if (keep_cum) {
                    cum[m][0] = f2_mul(cum[m][0], ww.x);
                    cum[m][1] = f2_mul(cum[m][1], ww.y);
                }
            }
#pragma unroll
            for (int c = 0; c < C; c++) {
                float lo, hi;
                f2_unpack(acc[c], lo, hi);
                p[u][c] = lo + hi;
            }
        }
        // the sums over the LI lanes of the column group, a fixed tree: while a lane holds several columns, each step
        // halves them; with one column left the steps are plain
        int first = 0;          // first column this lane still holds
        int nc = C, plain_bits = 0;
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
                if (up) first += hf;
                nc = hf;
            } else {
#pragma unroll
                for (int u = 0; u < U; u++) p[u][0] += __shfl_xor_sync(0xffffffffu, p[u][0], o);
                plain_bits |= o;
            }
        }
        // lanes that differ only in the bits of the plain steps hold the same sum: one of them writes
        if ((lane & plain_bits) == 0) {
#pragma unroll
            for (int u = 0; u < U; u++) {
                float* orow = a.out + (size_t)(t + u) * a.nh * dv + (size_t)h * dv + j0 + jl + first;
                const float* vp = rowp + u * ROW + V_AT + jl + first;
                const float bonus = rowp[u * ROW + B_AT];
#pragma unroll
                for (int c = 0; c < C; c++)
                    if (c < nc && j0 + jl + first + c < dv) {
                        if (PASS == 0) orow[c] = fmaf(bonus, vp[c], p[u][c]);
                        else orow[c] += p[u][c];
                    }
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
    if (PASS == 0) {
        store_state(P > 1 ? seg_base + seg * seg_stride : Sg);
        if (P > 1 && blockIdx.z == 0 && warp == 0 && lane < LI) {
            float* dst = dec_base + seg * dec_stride;
#pragma unroll
            for (int m = 0; m < M; m++) {
                const int i = m * 4 * LI + 4 * g;
                float v[4];
                f2_unpack(cum[m][0], v[0], v[1]);
                f2_unpack(cum[m][1], v[2], v[3]);
#pragma unroll
                for (int r = 0; r < 4; r++)
                    if (i + r < d) dst[i + r] = v[r];
            }
        }
    } else if (last_seg) {
        // the sequence's state: what came in, decayed over this segment, plus what the segment added
        load_state(seg_base + seg * seg_stride, dec_base + seg * dec_stride, true);
        store_state(Sg);
    }
}

// head sizes up to 1024 (the rows of a column group over at most 32 lanes), any value size
extern "C" int illm_wkv_supported(int d, int dv) { return d > 0 && d <= 1024 && dv > 0 ? 1 : 0; }

template <int R, int C, int LI>
static void wkv_scan_launch(WkvScanArgs a, int B, cudaStream_t s) {
    constexpr int DP = R * LI, JB = C * (32 / LI) * (WS_THREADS / 32), ROW = 3 * DP + JB + 4;
    int tile = (int)(48 * 1024 / sizeof(float) / (2 * ROW));
    a.tile = tile > WS_MAX_TILE ? WS_MAX_TILE : (tile < 1 ? 1 : tile);
    if (a.tile > WS_U) a.tile -= a.tile % WS_U;
    const size_t smem = (size_t)2 * a.tile * ROW * sizeof(float);
    const dim3 grid(B * a.segments, a.nh, (a.dv + JB - 1) / JB);
    illm_launch(wkv_scan_kernel<R, C, LI, 0>, grid, dim3(WS_THREADS), smem, s, a);
    if (a.segments > 1) illm_launch(wkv_scan_kernel<R, C, LI, 1>, grid, dim3(WS_THREADS), smem, s, a);
}

// y: the projections [T, ld] with r, k, v and the decay's inner products z at their offsets; w2 [nh * d, rank] (w2_dtype), w0, u
// float32 [nh * d].  Scratch: w [T, nh * d], bonus [T, nh]; with segments > 1 seg_state [B, segments, nh, dv, d] and seg_decay
// [B, segments, nh, d].  out: float32 [T, nh * dv].
extern "C" int illm_wkv_scan(const float* y, int T, int ld, int r_off, int k_off, int v_off, int z_off, int rank, int nh, int d, int dv, const void* w2,
                             int w2_dtype, const float* w0, const float* u, float* state, long long state_stride, const int* slots, const int* cu_q,
                             float* w, float* bonus, float* out, int B, int segments, float* seg_state, float* seg_decay, void* stream) {
    if (B <= 0 || T <= 0) return 0;
    if (segments < 1 || (segments > 1 && (!seg_state || !seg_decay)) || (long long)B * segments > 0x7fffffff) return ILLM_ERR_BAD_ARG;
    if (nh <= 0 || nh > 65535 || d <= 0 || d > 1024 || dv <= 0 || rank <= 0 || !y || !w2 || !w0 || !u || !state || !w || !bonus || !out ||
        state_stride < (long long)nh * d * dv)
        return ILLM_ERR_BAD_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    WkvPrepArgs p{y, T, ld, r_off, k_off, z_off, rank, nh, d, w0, u, w, bonus};
    const dim3 pgrid((T + WP_TOK - 1) / WP_TOK, nh);
    if (w2_dtype == ILLM_BF16) illm_launch(wkv_prep_kernel<bf16>, pgrid, dim3(128), 0, s, p, (const bf16*)w2);
    else if (w2_dtype == ILLM_F32) illm_launch(wkv_prep_kernel<float>, pgrid, dim3(128), 0, s, p, (const float*)w2);
    else return ILLM_ERR_BAD_ARG;
    WkvScanArgs a{y, ld, r_off, k_off, v_off, nh, d, dv, w, bonus, state, state_stride, slots, cu_q, out, 0, 0, segments, seg_state, seg_decay};
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
