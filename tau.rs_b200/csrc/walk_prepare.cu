// What the walks over a matrix state read, made in place from the projections in 32-bit, rows any distance apart:
//
//   forget gates:    queries pass SiLU; f = l + (1 - l) sigmoid(x) per head and channel, l a lower bound per channel
//   turned heads:    in every head of a row the first `rotary` elements are turned (element i with element i + rotary / 2, by the angle
//                    position * frequency[i]); heads from `scaled_from` on (the keys behind the queries) are multiplied by `scale`
#include "common.cuh"

namespace {

constexpr int kThreads = 256;

// grid (tokens, blocks of columns): the queries' columns first, then the gates'.
__global__ void __launch_bounds__(kThreads)
forget_gates_kernel(float* __restrict__ rows, long long stride, int query_offset, int gate_offset, const float* __restrict__ lower, int width) {
    grid_dependents_launch();
    grid_dependency_wait();
    const int column = blockIdx.y * kThreads + threadIdx.x;
    if (column >= width) return;
    float* row = rows + static_cast<size_t>(blockIdx.x) * stride;
    const float q = row[query_offset + column], x = row[gate_offset + column], l = lower[column];
    row[query_offset + column] = q / (1.0f + expf(-q));
    row[gate_offset + column] = l + (1.0f - l) / (1.0f + expf(-x));
}

// grid (tokens, blocks of items); an item is one pair, or one element that passes, of one head.
__global__ void __launch_bounds__(kThreads)
turn_heads_kernel(float* __restrict__ rows, long long stride, const int* __restrict__ positions, const float* __restrict__ frequency, int rotary,
                  int heads, int dim, int scaled_from, float scale) {
    grid_dependents_launch();
    grid_dependency_wait();
    const int half = rotary / 2, per_head = half + (dim - rotary);
    const int item = blockIdx.y * kThreads + threadIdx.x;
    if (item >= heads * per_head) return;
    const int head = item / per_head, within = item % per_head;
    const float factor = head >= scaled_from ? scale : 1.0f;
    float* from = rows + static_cast<size_t>(blockIdx.x) * stride + head * dim;
    if (within < half) {
        float sine, cosine;
        sincosf(static_cast<float>(positions[blockIdx.x]) * frequency[within], &sine, &cosine);
        const float u = from[within], v = from[within + half];
        from[within] = (u * cosine - v * sine) * factor;
        from[within + half] = (v * cosine + u * sine) * factor;
    } else {
        from[half + within] *= factor;
    }
}

}  // namespace

// In place on rows `stride` floats apart: columns [query_offset, + width) pass SiLU, columns [gate_offset, + width) become forget gates.
TAU_EXPORT int tau_forget_gates(float* rows, long long stride, int query_offset, int gate_offset, const float* lower, long long tokens, int width, void* stream) {
    if (tokens <= 0) return 0;
    if (!rows || !lower || width <= 0 || tokens > 0x7fffffffLL || query_offset < 0 || gate_offset < 0 || query_offset + width > stride || gate_offset + width > stride)
        return cudaErrorInvalidValue;
    tau_launch(forget_gates_kernel, dim3(static_cast<unsigned>(tokens), (width + kThreads - 1) / kThreads), dim3(kThreads), 0, static_cast<cudaStream_t>(stream), rows,
               stride, query_offset, gate_offset, lower, width);
    return tau_launch_status();
}

// In place on the first heads * dim columns of rows `stride` floats apart.
TAU_EXPORT int tau_turn_heads(float* rows, long long stride, const int* positions, const float* frequency, int rotary, long long tokens, int heads, int dim,
                              int scaled_from, float scale, void* stream) {
    if (tokens <= 0) return 0;
    if (!rows || !positions || heads <= 0 || dim <= 0 || rotary < 0 || rotary > dim || rotary % 2 != 0 || (rotary && !frequency) || tokens > 0x7fffffffLL ||
        static_cast<long long>(heads) * dim > stride)
        return cudaErrorInvalidValue;
    const int items = heads * (rotary / 2 + dim - rotary);
    tau_launch(turn_heads_kernel, dim3(static_cast<unsigned>(tokens), (items + kThreads - 1) / kThreads), dim3(kThreads), 0, static_cast<cudaStream_t>(stream), rows,
               stride, positions, frequency, rotary, heads, dim, scaled_from, scale);
    return tau_launch_status();
}
