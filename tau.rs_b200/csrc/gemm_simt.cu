// Plain tiled matrix product on the ordinary 32-bit pipes: out[M, N] = x[M, K] * w[N, K]^T + bias.
//
// This is the true 32-bit product (fused multiply-add in float, no tensor cores, no reduced-precision
// mode) and the fallback for bfloat16 shapes that the tensor-core kernels refuse.  The weight is the
// checkpoint's `[out, in]` matrix used as it lies (crates/cuda-kernels/src/kernels/
// linear_bf16_fp32.cuh:31-33).  Any M, N, K.
#include "common.cuh"

namespace {

constexpr int kTile = 64;     // output tile is kTile x kTile
constexpr int kDepth = 16;    // K elements per stage
constexpr int kThreads = 256; // each thread owns a 4 x 4 patch

template <typename TIn, typename TOut>
__global__ void __launch_bounds__(kThreads)
gemm_simt_kernel(const TIn* __restrict__ x, const TIn* __restrict__ w, const float* __restrict__ bias,
                 TOut* __restrict__ out, int M, int N, int K, long long x_stride, long long w_stride,
                 long long out_stride, long long x_batch, long long w_batch, long long out_batch) {
    grid_dependents_launch();
    grid_dependency_wait();
    // blockIdx.z numbers the products of a batch (one per head, say); each has its operands a fixed distance further on.
    x += blockIdx.z * x_batch;
    w += blockIdx.z * w_batch;
    out += blockIdx.z * out_batch;
    __shared__ float xs[kDepth][kTile + 4];
    __shared__ float ws[kDepth][kTile + 4];
    const int row0 = blockIdx.y * kTile, col0 = blockIdx.x * kTile;
    const int tx = threadIdx.x % 16, ty = threadIdx.x / 16;
    float acc[4][4] = {};
    // Loading: thread t brings element (t / 16 + 16 * i, t % 16) of each 64 x 16 tile, i = 0..3.
    const int load_k = threadIdx.x % kDepth, load_r = threadIdx.x / kDepth;
    for (int k0 = 0; k0 < K; k0 += kDepth) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int r = load_r + 16 * i;
            const int k = k0 + load_k;
            const int xr = row0 + r, wr = col0 + r;
            xs[load_k][r] = (xr < M && k < K) ? to_float(x[xr * x_stride + k]) : 0.0f;
            ws[load_k][r] = (wr < N && k < K) ? to_float(w[wr * w_stride + k]) : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < kDepth; ++k) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) a[i] = xs[k][ty * 4 + i];
#pragma unroll
            for (int j = 0; j < 4; ++j) b[j] = ws[k][tx * 4 + j];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int r = row0 + ty * 4 + i;
        if (r >= M) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int c = col0 + tx * 4 + j;
            if (c >= N) continue;
            const float value = acc[i][j] + (bias ? bias[c] : 0.0f);
            out[r * out_stride + c] = from_float<TOut>(value);
        }
    }
}

template <typename TIn, typename TOut>
int launch(const void* x, const void* w, const float* bias, void* out, int M, int N, int K, long long x_stride,
           long long w_stride, long long out_stride, cudaStream_t stream, int batch = 1, long long x_batch = 0, long long w_batch = 0,
           long long out_batch = 0) {
    dim3 grid((N + kTile - 1) / kTile, (M + kTile - 1) / kTile, batch);
    tau_launch(gemm_simt_kernel<TIn, TOut>, dim3(grid), dim3(kThreads), 0, stream, static_cast<const TIn*>(x), static_cast<const TIn*>(w), bias,
                                                              static_cast<TOut*>(out), M, N, K, x_stride, w_stride, out_stride, x_batch, w_batch, out_batch);
    return tau_launch_status();
}

// The batched product for few rows (single tokens against one small weight per head), bound by reading the weights once: a group of
// `kLanes` lanes takes a weight row in 16-byte pieces against up to eight rows of x, which lie in shared memory as floats.
// grid: (ceil(N / features_per_block), batch, ceil(M / 8)).
constexpr int kFewRows = 8;

template <typename TIn> struct Piece;
template <> struct Piece<bf16> { static constexpr int n = 8; };
template <> struct Piece<float> { static constexpr int n = 4; };
__device__ __forceinline__ void unpack_piece(const uint4& raw, float (&v)[8]) {
    const unsigned words[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        v[2 * i] = __uint_as_float(words[i] << 16);
        v[2 * i + 1] = __uint_as_float(words[i] & 0xffff0000u);
    }
}
__device__ __forceinline__ void unpack_piece(const uint4& raw, float (&v)[4]) {
    v[0] = __uint_as_float(raw.x); v[1] = __uint_as_float(raw.y); v[2] = __uint_as_float(raw.z); v[3] = __uint_as_float(raw.w);
}

template <typename TIn, typename TOut, int kLanes>
__global__ void __launch_bounds__(kThreads)
gemm_few_rows_kernel(const TIn* __restrict__ x, const TIn* __restrict__ w, TOut* __restrict__ out, int M, int N, int K, long long x_stride, long long w_stride,
                     long long out_stride, long long x_batch, long long w_batch, long long out_batch, int features_per_block) {
    grid_dependents_launch();
    grid_dependency_wait();
    constexpr int n = Piece<TIn>::n;
    extern __shared__ __align__(16) float rows[];      // [kFewRows][K]
    const int first_row = blockIdx.z * kFewRows, count = min(kFewRows, M - first_row);
    x += blockIdx.y * x_batch;
    w += blockIdx.y * w_batch;
    out += blockIdx.y * out_batch;
    for (int item = threadIdx.x; item < kFewRows * K; item += blockDim.x) {
        const int r = item / K;
        rows[item] = r < count ? to_float(x[(first_row + r) * x_stride + item - r * K]) : 0.0f;
    }
    __syncthreads();
    const int group = threadIdx.x / kLanes, lane = threadIdx.x % kLanes, groups = blockDim.x / kLanes;
    const int begin = blockIdx.x * features_per_block, end = min(N, begin + features_per_block);
    for (int base = begin; base < end; base += groups) {      // every lane of a warp takes every turn: they meet in the shuffles
        const int feature = base + group;
        float sums[kFewRows] = {};
        if (feature < end) {
            const TIn* weights = w + feature * w_stride;
            for (int column = lane * n; column < K; column += kLanes * n) {
                float v[n];
                unpack_piece(*reinterpret_cast<const uint4*>(weights + column), v);
#pragma unroll
                for (int r = 0; r < kFewRows; ++r) {
#pragma unroll
                    for (int i = 0; i < n; i += 4) {
                        const float4 a = *reinterpret_cast<const float4*>(rows + r * K + column + i);
                        sums[r] = fmaf(v[i], a.x, fmaf(v[i + 1], a.y, fmaf(v[i + 2], a.z, fmaf(v[i + 3], a.w, sums[r]))));
                    }
                }
            }
        }
#pragma unroll
        for (int r = 0; r < kFewRows; ++r)
#pragma unroll
            for (int offset = kLanes / 2; offset > 0; offset >>= 1) sums[r] += __shfl_xor_sync(0xffffffffu, sums[r], offset);
        if (feature < end) {
#pragma unroll
            for (int r = 0; r < kFewRows; ++r)
                if (r < count && lane == r % kLanes) out[(first_row + r) * out_stride + feature] = from_float<TOut>(sums[r]);
        }
    }
}

template <typename TIn, typename TOut>
int launch_few_rows(const void* x, const void* w, void* out, int M, int N, int K, long long x_stride, long long w_stride, long long out_stride, cudaStream_t stream,
                    int batch, long long x_batch, long long w_batch, long long out_batch) {
    const int lanes = K / Piece<TIn>::n <= 8 ? 8 : K / Piece<TIn>::n <= 16 ? 16 : 32;
    int features = 64;                              // smaller tiles while they leave SMs without a block
    while (features > kThreads / lanes && batch * ((N + features - 1) / features) < 2 * 148) features /= 2;
    const dim3 grid((N + features - 1) / features, batch, (M + kFewRows - 1) / kFewRows);
    const size_t bytes = static_cast<size_t>(kFewRows) * K * sizeof(float);
    auto* kernel = lanes == 8 ? gemm_few_rows_kernel<TIn, TOut, 8> : lanes == 16 ? gemm_few_rows_kernel<TIn, TOut, 16> : gemm_few_rows_kernel<TIn, TOut, 32>;
    tau_launch(kernel, grid, dim3(kThreads), bytes, stream, static_cast<const TIn*>(x), static_cast<const TIn*>(w), static_cast<TOut*>(out), M, N, K, x_stride, w_stride,
               out_stride, x_batch, w_batch, out_batch, features);
    return tau_launch_status();
}

template <typename TIn, typename TOut>
int launch_batched(const void* x, const void* w, void* out, int M, int N, int K, long long x_stride, long long w_stride, long long out_stride, cudaStream_t stream,
                   int batch, long long x_batch, long long w_batch, long long out_batch) {
    constexpr int n = Piece<TIn>::n;
    const bool few = M <= 2 * kFewRows && K % n == 0 && w_stride % n == 0 && w_batch % n == 0 && (reinterpret_cast<uintptr_t>(w) & 15) == 0
                     && static_cast<size_t>(kFewRows) * K * sizeof(float) <= 48 * 1024;
    if (few) return launch_few_rows<TIn, TOut>(x, w, out, M, N, K, x_stride, w_stride, out_stride, stream, batch, x_batch, w_batch, out_batch);
    return launch<TIn, TOut>(x, w, nullptr, out, M, N, K, x_stride, w_stride, out_stride, stream, batch, x_batch, w_batch, out_batch);
}

}  // namespace

// Strides are in elements between consecutive rows.  `out_dtype` may be float32 for a bfloat16 product (logits).
TAU_EXPORT int tau_gemm_simt(int in_dtype, int out_dtype, const void* x, const void* w, const float* bias, void* out, int M,
                             int N, int K, long long x_stride, long long w_stride, long long out_stride, void* stream) {
    if (M <= 0 || N <= 0) return 0;
    if (!x || !w || !out || K <= 0) return cudaErrorInvalidValue;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (in_dtype == TAU_F32 && out_dtype == TAU_F32) return launch<float, float>(x, w, bias, out, M, N, K, x_stride, w_stride, out_stride, s);
    if (in_dtype == TAU_BF16 && out_dtype == TAU_BF16) return launch<bf16, bf16>(x, w, bias, out, M, N, K, x_stride, w_stride, out_stride, s);
    if (in_dtype == TAU_BF16 && out_dtype == TAU_F32) return launch<bf16, float>(x, w, bias, out, M, N, K, x_stride, w_stride, out_stride, s);
    return cudaErrorInvalidValue;
}

// `batch` products of the same sizes in one launch: product b reads x + b * x_batch and w + b * w_batch and writes out + b * out_batch
// (elements).  No bias.
TAU_EXPORT int tau_gemm_simt_batched(int in_dtype, int out_dtype, const void* x, const void* w, void* out, int M, int N, int K, long long x_stride,
                                     long long w_stride, long long out_stride, int batch, long long x_batch, long long w_batch, long long out_batch,
                                     void* stream) {
    if (M <= 0 || N <= 0 || batch <= 0) return 0;
    if (!x || !w || !out || K <= 0 || batch > 65535) return cudaErrorInvalidValue;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (in_dtype == TAU_F32 && out_dtype == TAU_F32) return launch_batched<float, float>(x, w, out, M, N, K, x_stride, w_stride, out_stride, s, batch, x_batch, w_batch, out_batch);
    if (in_dtype == TAU_BF16 && out_dtype == TAU_BF16) return launch_batched<bf16, bf16>(x, w, out, M, N, K, x_stride, w_stride, out_stride, s, batch, x_batch, w_batch, out_batch);
    if (in_dtype == TAU_BF16 && out_dtype == TAU_F32) return launch_batched<bf16, float>(x, w, out, M, N, K, x_stride, w_stride, out_stride, s, batch, x_batch, w_batch, out_batch);
    return cudaErrorInvalidValue;
}
