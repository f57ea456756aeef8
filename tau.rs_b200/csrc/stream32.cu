// A residual stream kept in 32-bit beside activations of another dtype: embedding rows widened to float, and the
// fused sum of up to two branches into the stream followed by RMSNorm, with the output in the activations' dtype.
// Also the gated output stage of mixers whose result is 32-bit: optional RMS norm per group, weight, sigmoid gate; the same sum
// followed by an element-wise tanh in a norm's place; and a soft cap on logits.
#include "common.cuh"

namespace {

constexpr int kThreads = 256;

__device__ __forceinline__ float load_as_float(const void* base, int code, size_t index) {
    return code == TAU_BF16 ? __bfloat162float(static_cast<const bf16*>(base)[index]) : static_cast<const float*>(base)[index];
}

template <typename T>
__global__ void embedding_f32_kernel(const int* __restrict__ tokens, const T* __restrict__ table, float* __restrict__ out, int width, int vocab, float scale) {
    grid_dependents_launch();
    grid_dependency_wait();
    const int row = blockIdx.x;
    const int token = tokens[row];
    float* target = out + static_cast<size_t>(row) * width;
    const bool inside = token >= 0 && token < vocab;   // refused on the host already; never read outside the table
    const T* source = table + static_cast<size_t>(inside ? token : 0) * width;
    for (int column = threadIdx.x; column < width; column += blockDim.x) target[column] = inside ? to_float(source[column]) * scale : 0.0f;
}

// What joins a row of the stream: up to two branches, the factors on their sum (one number, and one per channel if there is a vector), and
// a row of a table (row table_ids[r] of `table_rows` rows, times `table_scale`), which no other factor touches.
struct Joining {
    const void* a;
    const void* b;
    const float* channel_scale;
    const void* table;
    const int* table_ids;
    int a_code, b_code, table_code, table_rows;
    float branch_scale, table_scale;
};

__device__ __forceinline__ bool anything_joins(const Joining& j) { return j.a != nullptr || j.table != nullptr; }

// The table's row that joins row r of the stream (nothing is read of a table whose row number lies outside it).
__device__ __forceinline__ long long table_row_of(const Joining& j, int r) {
    if (!j.table) return -1;
    const int id = j.table_ids[r];
    return id >= 0 && id < j.table_rows ? id : -1;
}

// r = rows ? rows[i] : i.  sum = stream[r] + branch_scale * channel_scale * (a[r] + b[r]) + table_scale * table[ids[r]] in 32-bit; if
// `update` the sum replaces stream[r]; out[i] = sum / sqrt(mean(sum^2) + eps) * weight, rounded once to T.  With `groups` > 1 the row is cut
// into that many equal consecutive pieces and each is divided by its own root mean square (a warp sums a piece's squares).
constexpr int kMaxNormGroups = 1024;

template <typename T>
__global__ void __launch_bounds__(kThreads)
stream_add_norm_kernel(float* __restrict__ stream, const Joining join, const int* __restrict__ rows, const float* __restrict__ weight,
                       T* __restrict__ out, int width, float eps, int update, int groups) {
    grid_dependents_launch();
    grid_dependency_wait();
    __shared__ float scratch[33];
    __shared__ float inverses[kMaxNormGroups];
    const int row = rows ? rows[blockIdx.x] : blockIdx.x;
    const size_t base = static_cast<size_t>(row) * width;
    const bool a = anything_joins(join);
    const long long table_row = table_row_of(join, row);
    auto joined = [&](int column) {
        float value = stream[base + column];
        if (join.a) {
            float branch = load_as_float(join.a, join.a_code, base + column);
            if (join.b) branch += load_as_float(join.b, join.b_code, base + column);
            if (join.channel_scale) branch *= join.channel_scale[column];
            value = fmaf(join.branch_scale, branch, value);
        }
        if (table_row >= 0) value = fmaf(join.table_scale, load_as_float(join.table, join.table_code, static_cast<size_t>(table_row) * width + column), value);
        return value;
    };
    T* target = out + static_cast<size_t>(blockIdx.x) * width;
    if (groups > 1) {
        if (update && a) {
            for (int column = threadIdx.x; column < width; column += blockDim.x) stream[base + column] = joined(column);
            __syncthreads();      // the pieces below are summed by other threads than those that wrote them
        }
        const bool stored = update || !a;
        const int piece = width / groups, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
        for (int group = warp; group < groups; group += warps) {
            float squares = 0.0f;
            for (int column = group * piece + lane; column < (group + 1) * piece; column += 32) {
                const float value = stored ? stream[base + column] : joined(column);
                squares = fmaf(value, value, squares);
            }
            squares = warp_sum(squares);
            if (lane == 0) inverses[group] = 1.0f / sqrtf(squares / static_cast<float>(piece) + eps);
        }
        __syncthreads();
        for (int column = threadIdx.x; column < width; column += blockDim.x)
            target[column] = from_float<T>((stored ? stream[base + column] : joined(column)) * inverses[column / piece] * weight[column]);
        return;
    }
    float squares = 0.0f;
    for (int column = threadIdx.x; column < width; column += blockDim.x) {
        const float value = joined(column);
        if (update) stream[base + column] = value;
        squares += value * value;
    }
    const float inverse = 1.0f / sqrtf(block_sum(squares, scratch) / static_cast<float>(width) + eps);
    for (int column = threadIdx.x; column < width; column += blockDim.x) {
        const float value = (a && !update) ? joined(column) : stream[base + column];     // each thread reads back what it wrote itself
        target[column] = from_float<T>(value * inverse * weight[column]);
    }
}

// r = rows ? rows[i] : i.  sum = stream[r] + branch_scale * (a[r] + b[r]) in 32-bit; if `update` the sum replaces stream[r];
// out[i] = tanh(alpha * sum) * weight + bias, rounded once to T.  No element needs another, so a thread takes `kPer` neighbouring columns
// of one row (16-byte accesses of the stream where kPer is 4).
template <int kPer>
__device__ __forceinline__ void load_columns(const void* base, int code, size_t index, float (&v)[kPer]) {
    if (kPer == 4 && code == TAU_BF16) {
        const uint2 raw = *reinterpret_cast<const uint2*>(static_cast<const bf16*>(base) + index);
        v[0] = __uint_as_float(raw.x << 16), v[1 % kPer] = __uint_as_float(raw.x & 0xffff0000u);
        v[2 % kPer] = __uint_as_float(raw.y << 16), v[3 % kPer] = __uint_as_float(raw.y & 0xffff0000u);
    } else if (kPer == 4) {
        const float4 raw = *reinterpret_cast<const float4*>(static_cast<const float*>(base) + index);
        v[0] = raw.x, v[1 % kPer] = raw.y, v[2 % kPer] = raw.z, v[3 % kPer] = raw.w;
    } else {
        v[0] = load_as_float(base, code, index);
    }
}

template <int kPer>
__device__ __forceinline__ void store_columns(float* target, const float (&v)[kPer]) {
    if (kPer == 4) *reinterpret_cast<float4*>(target) = make_float4(v[0], v[1 % kPer], v[2 % kPer], v[3 % kPer]);
    else target[0] = v[0];
}
template <int kPer>
__device__ __forceinline__ void store_columns(bf16* target, const float (&v)[kPer]) {
    if (kPer == 4) {
        const __nv_bfloat162 low = __floats2bfloat162_rn(v[0], v[1 % kPer]), high = __floats2bfloat162_rn(v[2 % kPer], v[3 % kPer]);
        *reinterpret_cast<uint2*>(target) = make_uint2(*reinterpret_cast<const unsigned*>(&low), *reinterpret_cast<const unsigned*>(&high));
    } else {
        target[0] = __float2bfloat16_rn(v[0]);
    }
}

// The same sum and norm (one group) for rows of whole 16-byte pieces: a thread holds its columns of the sum in registers between the two
// passes, four neighbouring ones at a time, `kPieces` times; width <= 4 * blockDim.x * kPieces.
template <typename T, int kPieces>
__global__ void __launch_bounds__(kThreads)
stream_add_norm_vec_kernel(float* __restrict__ stream, const Joining join, const int* __restrict__ rows, const float* __restrict__ weight,
                           T* __restrict__ out, int width, float eps, int update) {
    grid_dependents_launch();
    grid_dependency_wait();
    __shared__ float scratch[33];
    const int row = rows ? rows[blockIdx.x] : blockIdx.x;
    const size_t base = static_cast<size_t>(row) * width;
    const long long table_row = table_row_of(join, row);
    const bool store = update && anything_joins(join);
    float sum[kPieces][4];
    float squares = 0.0f;
#pragma unroll
    for (int piece = 0; piece < kPieces; ++piece) {
        const int column = (piece * blockDim.x + threadIdx.x) * 4;
        if (column >= width) break;
        load_columns<4>(stream, TAU_F32, base + column, sum[piece]);
        if (join.a) {
            float branch[4], other[4];
            load_columns<4>(join.a, join.a_code, base + column, branch);
            if (join.b) {
                load_columns<4>(join.b, join.b_code, base + column, other);
#pragma unroll
                for (int i = 0; i < 4; ++i) branch[i] += other[i];
            }
            if (join.channel_scale) {
                load_columns<4>(join.channel_scale, TAU_F32, column, other);
#pragma unroll
                for (int i = 0; i < 4; ++i) branch[i] *= other[i];
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) sum[piece][i] = fmaf(join.branch_scale, branch[i], sum[piece][i]);
        }
        if (table_row >= 0) {
            float looked_up[4];
            load_columns<4>(join.table, join.table_code, static_cast<size_t>(table_row) * width + column, looked_up);
#pragma unroll
            for (int i = 0; i < 4; ++i) sum[piece][i] = fmaf(join.table_scale, looked_up[i], sum[piece][i]);
        }
        if (store) store_columns<4>(stream + base + column, sum[piece]);
#pragma unroll
        for (int i = 0; i < 4; ++i) squares = fmaf(sum[piece][i], sum[piece][i], squares);
    }
    const float inverse = 1.0f / sqrtf(block_sum(squares, scratch) / static_cast<float>(width) + eps);
    T* target = out + static_cast<size_t>(blockIdx.x) * width;
#pragma unroll
    for (int piece = 0; piece < kPieces; ++piece) {
        const int column = (piece * blockDim.x + threadIdx.x) * 4;
        if (column >= width) break;
        float w[4], result[4];
        load_columns<4>(weight, TAU_F32, column, w);
#pragma unroll
        for (int i = 0; i < 4; ++i) result[i] = sum[piece][i] * inverse * w[i];
        store_columns<4>(target + column, result);
    }
}

template <typename T>
void launch_add_norm(float* stream_values, const Joining& join, const int* rows, const float* weight, void* out, int out_rows, int width, float eps, int update,
                     int groups, cudaStream_t s) {
    auto whole = [](const void* pointer) { return (reinterpret_cast<uintptr_t>(pointer) & 15u) == 0; };      // a null pointer is aligned
    const bool vectors = groups == 1 && width % 4 == 0 && width <= 4 * kThreads * 8 && whole(stream_values) && whole(join.a) && whole(join.b) && whole(join.channel_scale)
                         && whole(join.table) && whole(weight) && whole(out);
    if (!vectors) {
        tau_launch(stream_add_norm_kernel<T>, dim3(out_rows), dim3(kThreads), 0, s, stream_values, join, rows, weight, static_cast<T*>(out), width, eps, update, groups);
        return;
    }
    const int pieces = (width / 4 + kThreads - 1) / kThreads;      // of four columns to a thread
    const dim3 block(pieces == 1 ? (width / 4 + 31) / 32 * 32 : kThreads);
    auto* kernel = pieces == 1 ? stream_add_norm_vec_kernel<T, 1> : pieces == 2 ? stream_add_norm_vec_kernel<T, 2> : pieces <= 4 ? stream_add_norm_vec_kernel<T, 4> : stream_add_norm_vec_kernel<T, 8>;
    tau_launch(kernel, dim3(out_rows), block, 0, s, stream_values, join, rows, weight, static_cast<T*>(out), width, eps, update);
}

template <typename T, int kPer>
__global__ void __launch_bounds__(kThreads)
stream_add_tanh_kernel(float* __restrict__ stream, const void* __restrict__ a, int a_code, const void* __restrict__ b, int b_code, const int* __restrict__ rows,
                       const float* __restrict__ alpha, const float* __restrict__ weight, const float* __restrict__ bias, T* __restrict__ out, int width,
                       int update, float branch_scale) {
    grid_dependents_launch();
    grid_dependency_wait();
    const int column = (blockIdx.y * kThreads + threadIdx.x) * kPer;
    if (column >= width) return;
    const size_t base = static_cast<size_t>(rows ? rows[blockIdx.x] : static_cast<int>(blockIdx.x)) * width + column;
    float value[kPer], result[kPer];
    load_columns<kPer>(stream, TAU_F32, base, value);
    if (a) {
        float branch[kPer];
        load_columns<kPer>(a, a_code, base, branch);
        if (b) {
            float second[kPer];
            load_columns<kPer>(b, b_code, base, second);
#pragma unroll
            for (int i = 0; i < kPer; ++i) branch[i] += second[i];
        }
#pragma unroll
        for (int i = 0; i < kPer; ++i) value[i] = fmaf(branch_scale, branch[i], value[i]);
        if (update) store_columns<kPer>(stream + base, value);
    }
    float w[kPer], offset[kPer];
    load_columns<kPer>(weight, TAU_F32, column, w);
    load_columns<kPer>(bias, TAU_F32, column, offset);
    const float steep = *alpha;
#pragma unroll
    for (int i = 0; i < kPer; ++i) result[i] = fmaf(tanhf(steep * value[i]), w[i], offset[i]);
    store_columns<kPer>(out + static_cast<size_t>(blockIdx.x) * width + column, result);
}

template <typename T>
void launch_add_tanh(float* stream_values, const void* a, int a_code, const void* b, int b_code, const int* rows, const float* alpha, const float* weight,
                     const float* bias, void* out, int out_rows, int width, int update, float branch_scale, cudaStream_t s) {
    if (width % 4 == 0)
        tau_launch(stream_add_tanh_kernel<T, 4>, dim3(out_rows, (width / 4 + kThreads - 1) / kThreads), dim3(width / 4 < kThreads ? (width / 4 + 31) / 32 * 32 : kThreads), 0, s,
                   stream_values, a, a_code, b, b_code, rows, alpha, weight, bias, static_cast<T*>(out), width, update, branch_scale);
    else
        tau_launch(stream_add_tanh_kernel<T, 1>, dim3(out_rows, (width + kThreads - 1) / kThreads), dim3(kThreads), 0, s, stream_values, a, a_code, b, b_code,
                   rows, alpha, weight, bias, static_cast<T*>(out), width, update, branch_scale);
}

// logits = cap * tanh(logits / cap), in place.
template <int kPer>
__global__ void __launch_bounds__(kThreads) soft_cap_kernel(float* __restrict__ values, long long count, float cap) {
    grid_dependents_launch();
    grid_dependency_wait();
    for (long long index = (blockIdx.x * static_cast<long long>(kThreads) + threadIdx.x) * kPer; index < count; index += static_cast<long long>(gridDim.x) * kThreads * kPer) {
        float v[kPer];
        load_columns<kPer>(values, TAU_F32, index, v);
#pragma unroll
        for (int i = 0; i < kPer; ++i) v[i] = cap * tanhf(v[i] / cap);
        store_columns<kPer>(values + index, v);
    }
}

// out[row] = left_scale * left[row] / rms(left[row]) * left_weight + right_scale * right[row] / rms(right[row]) * right_weight: two results
// that are normalised over their whole width, each with its own weight, before they are added (eps inside the roots); all 32-bit.
__global__ void __launch_bounds__(kThreads)
normed_pair_sum_kernel(const float* __restrict__ left, const float* __restrict__ right, const float* __restrict__ left_weight,
                       const float* __restrict__ right_weight, float* __restrict__ out, int width, float eps, float left_scale, float right_scale) {
    grid_dependents_launch();
    grid_dependency_wait();
    __shared__ float scratch[33];
    const size_t base = static_cast<size_t>(blockIdx.x) * width;
    float a = 0.0f, b = 0.0f;
    for (int column = threadIdx.x; column < width; column += blockDim.x) {
        const float x = left[base + column], y = right[base + column];
        a = fmaf(x, x, a);
        b = fmaf(y, y, b);
    }
    const float left_factor = left_scale / sqrtf(block_sum(a, scratch) / static_cast<float>(width) + eps);
    const float right_factor = right_scale / sqrtf(block_sum(b, scratch) / static_cast<float>(width) + eps);
    for (int column = threadIdx.x; column < width; column += blockDim.x)
        out[base + column] = left[base + column] * left_factor * left_weight[column] + right[base + column] * right_factor * right_weight[column];
}

// values [rows, groups * group_width] in 32-bit.  With `normalize` each group of a row is divided by its root mean square;
// then times weight (if any), times sigmoid(gate) or, with `silu_gate`, gate * sigmoid(gate) (if any; gate rows lie `gate_stride`
// apart), rounded once to T; output rows lie `out_stride` apart.
template <typename T>
__global__ void __launch_bounds__(kThreads)
gated_group_norm_kernel(const float* __restrict__ values, const float* __restrict__ weight, const void* __restrict__ gate, int gate_code, long long gate_stride,
                        T* __restrict__ out, long long out_stride, int groups, int group_width, float eps, int normalize, int silu_gate) {
    grid_dependents_launch();
    grid_dependency_wait();
    const int row = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    const int width = groups * group_width;
    const float* source = values + static_cast<size_t>(row) * width;
    __shared__ float scratch[33];
    if (groups >= warps || gridDim.y > 1) {       // many groups: a warp takes a group at a time (of the row's share of this block)
        for (int group = blockIdx.y * warps + warp; group < groups; group += warps * gridDim.y) {
            float inverse = 1.0f;
            if (normalize) {
                float squares = 0.0f;
                for (int column = lane; column < group_width; column += 32) {
                    const float value = source[group * group_width + column];
                    squares += value * value;
                }
                inverse = 1.0f / sqrtf(warp_sum(squares) / static_cast<float>(group_width) + eps);
            }
            for (int column = lane; column < group_width; column += 32) {
                const int index = group * group_width + column;
                float value = source[index] * inverse;
                if (weight) value *= weight[index];
                if (gate) {
                    const float z = load_as_float(gate, gate_code, static_cast<size_t>(row) * gate_stride + index);
                    value *= (silu_gate ? z : 1.0f) / (1.0f + expf(-z));
                }
                out[static_cast<size_t>(row) * out_stride + index] = from_float<T>(value);
            }
        }
        return;
    }
    for (int group = 0; group < groups; ++group) {     // few groups: the whole block takes one after the other
        float inverse = 1.0f;
        if (normalize) {
            float squares = 0.0f;
            for (int column = threadIdx.x; column < group_width; column += blockDim.x) {
                const float value = source[group * group_width + column];
                squares += value * value;
            }
            inverse = 1.0f / sqrtf(block_sum(squares, scratch) / static_cast<float>(group_width) + eps);
        }
        for (int column = threadIdx.x; column < group_width; column += blockDim.x) {
            const int index = group * group_width + column;
            float value = source[index] * inverse;
            if (weight) value *= weight[index];
            if (gate) {
                const float z = load_as_float(gate, gate_code, static_cast<size_t>(row) * gate_stride + index);
                value *= (silu_gate ? z : 1.0f) / (1.0f + expf(-z));
            }
            out[static_cast<size_t>(row) * out_stride + index] = from_float<T>(value);
        }
    }
}

}  // namespace

TAU_EXPORT int tau_embedding_f32(int table_dtype, const int* tokens, const void* table, float* out, int rows, int width, int vocab, float scale, void* stream) {
    if (rows <= 0) return 0;
    if (!tokens || !table || !out || width <= 0 || vocab <= 0) return cudaErrorInvalidValue;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (table_dtype == TAU_F32) tau_launch(embedding_f32_kernel<float>, dim3(rows), dim3(kThreads), 0, s, tokens, static_cast<const float*>(table), out, width, vocab, scale);
    else if (table_dtype == TAU_BF16) tau_launch(embedding_f32_kernel<bf16>, dim3(rows), dim3(kThreads), 0, s, tokens, static_cast<const bf16*>(table), out, width, vocab, scale);
    else return cudaErrorInvalidValue;
    return tau_launch_status();
}

TAU_EXPORT int tau_stream_add_norm(int out_dtype, float* stream_values, const void* a, int a_dtype, const void* b, int b_dtype, const int* rows,
                                   const float* weight, void* out, int out_rows, int width, float eps, int update, int groups, float branch_scale,
                                   const float* channel_scale, const void* table, int table_dtype, int table_rows, const int* table_ids, float table_scale,
                                   void* stream) {
    if (out_rows <= 0) return 0;
    if (!stream_values || !weight || !out || width <= 0 || (b && !a) || (update && rows) || groups < 1 || groups > kMaxNormGroups || width % groups != 0
        || (table && (!table_ids || table_rows <= 0)) || (channel_scale && !a))
        return cudaErrorInvalidValue;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    const Joining join{a, b, channel_scale, table, table_ids, a_dtype, b_dtype, table_dtype, table_rows, branch_scale, table_scale};
    if (out_dtype == TAU_F32) launch_add_norm<float>(stream_values, join, rows, weight, out, out_rows, width, eps, update, groups, s);
    else if (out_dtype == TAU_BF16) launch_add_norm<bf16>(stream_values, join, rows, weight, out, out_rows, width, eps, update, groups, s);
    else return cudaErrorInvalidValue;
    return tau_launch_status();
}

TAU_EXPORT int tau_stream_add_tanh(int out_dtype, float* stream_values, const void* a, int a_dtype, const void* b, int b_dtype, const int* rows,
                                   const float* alpha, const float* weight, const float* bias, void* out, int out_rows, int width, int update,
                                   float branch_scale, void* stream) {
    if (out_rows <= 0) return 0;
    if (!stream_values || !alpha || !weight || !bias || !out || width <= 0 || (b && !a) || (update && rows)) return cudaErrorInvalidValue;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (out_dtype == TAU_F32) launch_add_tanh<float>(stream_values, a, a_dtype, b, b_dtype, rows, alpha, weight, bias, out, out_rows, width, update, branch_scale, s);
    else if (out_dtype == TAU_BF16) launch_add_tanh<bf16>(stream_values, a, a_dtype, b, b_dtype, rows, alpha, weight, bias, out, out_rows, width, update, branch_scale, s);
    else return cudaErrorInvalidValue;
    return tau_launch_status();
}

TAU_EXPORT int tau_soft_cap(float* values, long long count, float cap, void* stream) {
    if (count <= 0) return 0;
    if (!values || !(cap > 0.0f)) return cudaErrorInvalidValue;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    const bool vectors = count % 4 == 0 && (reinterpret_cast<uintptr_t>(values) & 15u) == 0;
    const long long blocks = (count / (vectors ? 4 : 1) + kThreads - 1) / kThreads;
    const dim3 grid(static_cast<unsigned>(blocks < 148 * 8 ? blocks : 148 * 8));
    if (vectors) tau_launch(soft_cap_kernel<4>, grid, dim3(kThreads), 0, s, values, count, cap);
    else tau_launch(soft_cap_kernel<1>, grid, dim3(kThreads), 0, s, values, count, cap);
    return tau_launch_status();
}

TAU_EXPORT int tau_normed_pair_sum(const float* left, const float* right, const float* left_weight, const float* right_weight, float* out, int rows, int width,
                                   float eps, float left_scale, float right_scale, void* stream) {
    if (rows <= 0) return 0;
    if (!left || !right || !left_weight || !right_weight || !out || width <= 0) return cudaErrorInvalidValue;
    tau_launch(normed_pair_sum_kernel, dim3(rows), dim3(kThreads), 0, static_cast<cudaStream_t>(stream), left, right, left_weight, right_weight, out, width, eps,
               left_scale, right_scale);
    return tau_launch_status();
}

TAU_EXPORT int tau_gated_group_norm(int dtype, const float* values, const float* weight, const void* gate, int gate_dtype, long long gate_stride, void* out, long long out_stride,
                                    int rows, int groups, int group_width, float eps, int normalize, int silu_gate, void* stream) {
    if (rows <= 0) return 0;
    if (!values || !out || groups <= 0 || group_width <= 0) return cudaErrorInvalidValue;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    // Few rows of many groups: a warp to a group, two warps to a block, so that a row's groups meet as many SMs as they can.
    const bool spread = groups > 1 && rows * 4 <= 148 * 2 && group_width <= 1024;
    const int threads = spread ? 64 : 256;
    const dim3 grid(rows, spread ? (groups + 1) / 2 : 1);
    if (dtype == TAU_F32) tau_launch(gated_group_norm_kernel<float>, grid, dim3(threads), 0, s, values, weight, gate, gate_dtype, gate_stride, static_cast<float*>(out), out_stride, groups, group_width, eps, normalize, silu_gate);
    else if (dtype == TAU_BF16) tau_launch(gated_group_norm_kernel<bf16>, grid, dim3(threads), 0, s, values, weight, gate, gate_dtype, gate_stride, static_cast<bf16*>(out), out_stride, groups, group_width, eps, normalize, silu_gate);
    else return cudaErrorInvalidValue;
    return tau_launch_status();
}
