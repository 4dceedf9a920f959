// The norm of a block whose sublayers read the stream as it is and whose outputs are normed on their way into it:
//
//   x[r] <- x[r] + y[r] / sqrt(mean(y[r]^2) + eps) * w;   h[r] = x[r] rounded to the compute dtype (optional)
//
// y is the sublayer's float32 output, finished or as the unreduced K slices of a split matrix product (float32
// [splits, rows, H], added in ascending order).  And, in front of such a block's first layer, the embedding's row through the
// same norm:
//
//   x[t] = e / sqrt(mean(e^2) + eps) * w,  e = table[ids[t]];   h[t] as above (an id outside the table: zeros, error word 1)
//
// Everything is float32 up to the rounding of h.  One block per row, a row's values in registers (four neighbouring
// channels per thread and piece) for rows of up to 16,384 channels that are a multiple of four, else in shared memory; the
// block's size and the order of the sums follow from the width alone, so a row's bits do not depend on the launch.
#include "common.cuh"

__device__ __forceinline__ void on_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void on_store4(bf16* p, float4 v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&lo), *reinterpret_cast<const unsigned*>(&hi));
}
__device__ __forceinline__ float4 on_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 on_load4(const bf16* p) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
    return make_float4(a.x, a.y, b.x, b.y);
}

template <int NV> __device__ __forceinline__ float on_inverse_rms(const float4* v, int H, float eps, float* scratch) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; i++) ss = fmaf(v[i].x, v[i].x, ss), ss = fmaf(v[i].y, v[i].y, ss), ss = fmaf(v[i].z, v[i].z, ss), ss = fmaf(v[i].w, v[i].w, ss);
    return 1.0f / sqrtf(block_sum(ss, scratch) / (float)H + eps);
}

template <typename TH, int NV>
__global__ void __launch_bounds__(512)
join_rmsnorm_kernel(float* __restrict__ x, const float* __restrict__ y, int splits, long long stride, const float* __restrict__ w, TH* __restrict__ h,
                    int H, float eps) {
    pdl_grid_sync();
    __shared__ float scratch[32];
    float* xr = x + (size_t)blockIdx.x * H;
    const float* yr = y + (size_t)blockIdx.x * H;
    float4 v[NV], xv[NV];
#pragma unroll
    for (int i = 0; i < NV; i++) {
        const int c = (threadIdx.x + i * blockDim.x) * 4;
        v[i] = c < H ? on_load4(yr + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        xv[i] = c < H ? on_load4(xr + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    constexpr int K = NV <= 4 ? 4 : 1;         // slices on their way at a time, added in their order
    for (int s = 1; s < splits; s += K) {
        float4 q[K][NV];
#pragma unroll
        for (int k = 0; k < K; k++)
#pragma unroll
            for (int i = 0; i < NV; i++) {
                const int c = (threadIdx.x + i * blockDim.x) * 4;
                q[k][i] = c < H && s + k < splits ? on_load4(yr + (size_t)(s + k) * stride + c) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
#pragma unroll
        for (int k = 0; k < K; k++)
#pragma unroll
            for (int i = 0; i < NV; i++) v[i].x += q[k][i].x, v[i].y += q[k][i].y, v[i].z += q[k][i].z, v[i].w += q[k][i].w;
    }
    const float inv = on_inverse_rms<NV>(v, H, eps, scratch);
#pragma unroll
    for (int i = 0; i < NV; i++) {
        const int c = (threadIdx.x + i * blockDim.x) * 4;
        if (c >= H) break;
        const float4 wv = on_load4(w + c);
        const float4 o = make_float4(xv[i].x + (v[i].x * inv) * wv.x, xv[i].y + (v[i].y * inv) * wv.y, xv[i].z + (v[i].z * inv) * wv.z,
                                     xv[i].w + (v[i].w * inv) * wv.w);
        on_store4(xr + c, o);
        if (h) on_store4(h + (size_t)blockIdx.x * H + c, o);
    }
}

// any width: the row in shared memory
template <typename TH>
__global__ void __launch_bounds__(256)
join_rmsnorm_any_kernel(float* __restrict__ x, const float* __restrict__ y, int splits, long long stride, const float* __restrict__ w, TH* __restrict__ h,
                        int H, float eps) {
    pdl_grid_sync();
    extern __shared__ float row[];
    __shared__ float scratch[32];
    float* xr = x + (size_t)blockIdx.x * H;
    const float* yr = y + (size_t)blockIdx.x * H;
    float ss = 0.f;
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        float v = yr[c];
        for (int s = 1; s < splits; s++) v += yr[(size_t)s * stride + c];
        row[c] = v;
        ss = fmaf(v, v, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)H + eps);
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        const float o = xr[c] + (row[c] * inv) * w[c];
        xr[c] = o;
        if (h) h[(size_t)blockIdx.x * H + c] = from_f32<TH>(o);
    }
}

template <typename TW, typename TH, int NV>
__global__ void __launch_bounds__(512)
embedding_normed_kernel(const int* __restrict__ ids, const TW* __restrict__ table, int V, const float* __restrict__ w, float* __restrict__ x,
                        TH* __restrict__ h, int H, float eps, int* __restrict__ err) {
    pdl_grid_sync();
    __shared__ float scratch[32];
    const int id = ids[blockIdx.x];
    const bool ok = id >= 0 && id < V;
    if (!ok && threadIdx.x == 0) atomicExch(err, 1);
    const TW* row = table + (size_t)(ok ? id : 0) * H;
    float4 v[NV];
#pragma unroll
    for (int i = 0; i < NV; i++) {
        const int c = (threadIdx.x + i * blockDim.x) * 4;
        v[i] = ok && c < H ? on_load4(row + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const float inv = on_inverse_rms<NV>(v, H, eps, scratch);
#pragma unroll
    for (int i = 0; i < NV; i++) {
        const int c = (threadIdx.x + i * blockDim.x) * 4;
        if (c >= H) break;
        const float4 wv = on_load4(w + c);
        const float4 o = make_float4((v[i].x * inv) * wv.x, (v[i].y * inv) * wv.y, (v[i].z * inv) * wv.z, (v[i].w * inv) * wv.w);
        on_store4(x + (size_t)blockIdx.x * H + c, o);
        if (h) on_store4(h + (size_t)blockIdx.x * H + c, o);
    }
}

template <typename TW, typename TH>
__global__ void __launch_bounds__(256)
embedding_normed_any_kernel(const int* __restrict__ ids, const TW* __restrict__ table, int V, const float* __restrict__ w, float* __restrict__ x,
                            TH* __restrict__ h, int H, float eps, int* __restrict__ err) {
    pdl_grid_sync();
    __shared__ float scratch[32];
    const int id = ids[blockIdx.x];
    const bool ok = id >= 0 && id < V;
    if (!ok && threadIdx.x == 0) atomicExch(err, 1);
    const TW* row = table + (size_t)(ok ? id : 0) * H;
    float ss = 0.f;
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        const float v = ok ? to_f32(row[c]) : 0.f;
        ss = fmaf(v, v, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)H + eps);
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        const float o = ((ok ? to_f32(row[c]) : 0.f) * inv) * w[c];
        x[(size_t)blockIdx.x * H + c] = o;
        if (h) h[(size_t)blockIdx.x * H + c] = from_f32<TH>(o);
    }
}

// threads of a row of H channels, and how many pieces of four channels a thread then holds (1, 2, 4 or 8; 0: too wide)
static int on_threads(int H) { return H <= 512 ? 128 : H <= 4096 ? 256 : 512; }
static int on_pieces(int H) {
    if (H % 4 || H > 16384) return 0;
    const int n = (H / 4 + on_threads(H) - 1) / on_threads(H);
    return n <= 1 ? 1 : n <= 2 ? 2 : n <= 4 ? 4 : 8;
}
#define ILLM_ON_PIECES(H, CALL)         \
    switch (on_pieces(H)) {             \
        case 1: CALL(1); break;         \
        case 2: CALL(2); break;         \
        case 4: CALL(4); break;         \
        default: CALL(8); break;        \
    }

// y: float32 [n_rows, H], splits of it `stride` floats apart; h (h_dtype) or nullptr
extern "C" int illm_join_rmsnorm(float* x, const float* y, int splits, long long stride, const float* w, void* h, int h_dtype, int n_rows, int H,
                                 float eps, void* stream) {
    if (n_rows <= 0) return 0;
    if (H <= 0 || !x || !y || !w || splits < 1) return ILLM_ERR_BAD_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    if (h && h_dtype != ILLM_F32 && h_dtype != ILLM_BF16) return ILLM_ERR_BAD_ARG;
    const bool half = h && h_dtype == ILLM_BF16;
    const bool vec = on_pieces(H) > 0 && !(((uintptr_t)x | (uintptr_t)y | (uintptr_t)w | (uintptr_t)h) & 15) && !(stride & 3);
    if (!vec) {
        const size_t smem = (size_t)H * sizeof(float);
        if (smem > 200 * 1024) return ILLM_ERR_BAD_ARG;
        if (half) {
            if (smem > 48 * 1024) cudaFuncSetAttribute(join_rmsnorm_any_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            illm_launch(join_rmsnorm_any_kernel<bf16>, dim3(n_rows), dim3(256), smem, s, x, y, splits, stride, w, (bf16*)h, H, eps);
        } else {
            if (smem > 48 * 1024) cudaFuncSetAttribute(join_rmsnorm_any_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            illm_launch(join_rmsnorm_any_kernel<float>, dim3(n_rows), dim3(256), smem, s, x, y, splits, stride, w, (float*)h, H, eps);
        }
        return illm_launch_status();
    }
#define ILLM_JOIN(NV)                                                                                                                             \
    do {                                                                                                                                          \
        if (half) illm_launch((join_rmsnorm_kernel<bf16, NV>), dim3(n_rows), dim3(on_threads(H)), 0, s, x, y, splits, stride, w, (bf16*)h, H, eps); \
        else illm_launch((join_rmsnorm_kernel<float, NV>), dim3(n_rows), dim3(on_threads(H)), 0, s, x, y, splits, stride, w, (float*)h, H, eps);    \
    } while (0)
    ILLM_ON_PIECES(H, ILLM_JOIN)
#undef ILLM_JOIN
    return illm_launch_status();
}

// x float32 [T, H]; h (h_dtype) or nullptr
extern "C" int illm_embedding_normed(const int* ids, const void* table, int table_dtype, const float* w, float* x, void* h, int h_dtype, int T, int H,
                                     int V, float eps, int* err, void* stream) {
    if (T <= 0) return 0;
    if (H <= 0 || V <= 0 || !table || !w || !x) return ILLM_ERR_BAD_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    const bool vec = on_pieces(H) > 0 && !(((uintptr_t)table | (uintptr_t)x | (uintptr_t)w | (uintptr_t)h) & 15);
#define ILLM_EN(TW, TH, NV)                                                                                                                       \
    do {                                                                                                                                          \
        if (NV) illm_launch((embedding_normed_kernel<TW, TH, (NV) ? (NV) : 1>), dim3(T), dim3(on_threads(H)), 0, s, ids, (const TW*)table, V, w, x, \
                            (TH*)h, H, eps, err);                                                                                                 \
        else illm_launch((embedding_normed_any_kernel<TW, TH>), dim3(T), dim3(256), 0, s, ids, (const TW*)table, V, w, x, (TH*)h, H, eps, err);    \
    } while (0)
    if (table_dtype == ILLM_BF16 && (!h || h_dtype == ILLM_BF16)) {
#define ILLM_ENB(NV) ILLM_EN(bf16, bf16, NV)
        if (!vec) ILLM_ENB(0);
        else ILLM_ON_PIECES(H, ILLM_ENB)
    } else if (table_dtype == ILLM_F32 && (!h || h_dtype == ILLM_F32)) {
#define ILLM_ENF(NV) ILLM_EN(float, float, NV)
        if (!vec) ILLM_ENF(0);
        else ILLM_ON_PIECES(H, ILLM_ENF)
    } else {
        return ILLM_ERR_BAD_ARG;
    }
#undef ILLM_EN
#undef ILLM_ENB
#undef ILLM_ENF
    return illm_launch_status();
}
