// Grouped-query softmax attention over cached rows for heads of any sizes, with the mask and the denominator as parameters:
//
//   * key and value sizes may differ (`dim`, `vdim`); one cached row per position holds [kv_heads x key | kv_heads x value], or keys
//     and values lie in pages of their own in the layout of ordinary heads, [pages, kv_heads, positions of a page, dim or vdim];
//   * a query at position i sees key j <= i if j > i - window (`window` > 0), or if j lies in i's chunk, floor(j / chunk) ==
//     floor(i / chunk) (`chunk` > 0; chunks are counted from position 0 of the sequence), or always (both 0); the sequence's first
//     `keep_first` positions stay visible however far back they lie;
//   * `talk` ([heads, heads]): the scores of all heads are mixed before the softmax, score_h <- sum_g talk[h, g] score_g.  A score is linear
//     in its query, so for runs of tokens prepare mixes the queries instead: head h asks every key head j with the query
//     sum over the heads g of j's group of talk[h, g] q_g, one query of kv_heads * dim elements against the position's keys of all key
//     heads side by side (`shared_keys`).  Single tokens take the kernel at the end of this file, which mixes the scores themselves;
//   * prepare may mix the values with another layer's of the same token, v <- (1 - share) v + share first;
//   * `sink`: the denominator of the softmax has exp(0) added (a key with score 0 and no value);
//   * the result is multiplied by `out_scale` before its one rounding; output rows may lie any distance apart;
//   * `distance` (two numbers r1, r2 per head): r1 * ln(1 + r2 * (i - j)) is taken off the score of key j for the query at i;
//   * `sigmoid_weights`: no softmax; a visible key weighs sigmoid(score + head_offset[head]) and the weights are not normalised;
//   * `gate`: the result is multiplied by sigmoid(gate), one number per (token, head) or one per element of the head's result;
//   * prepare may multiply the query at position p by 1 + coef * ln(floor((p + 1) / every) + 1) (a temperature that grows with the
//     position), and may be asked for the queries alone (a layer that reads the keys and values another layer cached).
//
//   prepare:    q and k divided by the root mean square over the WHOLE projection (all heads together; eps inside the root) and
//               multiplied by a weight of that size (or left as they are without weights); then in every head the first `rotary`
//               elements are turned: element i is paired with element i + rotary / 2, by the angle position * frequency[i], with
//               sine and cosine multiplied by `magnitude`; queries to [tokens, heads, dim], keys and values to the token's row.
//   attention:  a warp per (token, head): 32 keys at a time, a lane scores one key, then every lane sums its own value columns;
//               running maximum (never below the sink's 0 when there is one) and sum; scores, weights and sums in 32-bit.
#include "common.cuh"

namespace {

constexpr int kWarps = 8;
constexpr int kMaxShared = 224 * 1024;      // dynamic shared memory that a block of these kernels may ask for
constexpr int kMaxOwned = 16;     // value columns per lane: vdim <= 512

// The keys that a query sees, numbered 0 .. count - 1: the kept first positions that lie before its window (or chunk), then the window's.
struct Visible {
    int first, kept, count;
    __device__ __forceinline__ int key(int number) const { return number < kept ? number : first + number - kept; }
};
__device__ __forceinline__ Visible visible_keys(int position, int window, int chunk, int keep_first) {
    Visible seen;
    seen.first = 0;
    if (window > 0 && position - window + 1 > 0) seen.first = position - window + 1;
    if (chunk > 0) seen.first = position / chunk * chunk;
    seen.kept = keep_first < seen.first ? keep_first : seen.first;
    seen.count = seen.kept + position - seen.first + 1;
    return seen;
}

constexpr int kMixColumns = 8, kMixHeads = 4;      // of a thread where rows allow 16-byte accesses
__device__ __forceinline__ void load_columns(const float* source, float (&v)[kMixColumns]) {
    const float4 low = reinterpret_cast<const float4*>(source)[0], high = reinterpret_cast<const float4*>(source)[1];
    v[0] = low.x, v[1] = low.y, v[2] = low.z, v[3] = low.w, v[4] = high.x, v[5] = high.y, v[6] = high.z, v[7] = high.w;
}
__device__ __forceinline__ void load_columns(const bf16* source, float (&v)[kMixColumns]) {
    const uint4 raw = *reinterpret_cast<const uint4*>(source);
    const uint32_t words[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) v[2 * i] = __uint_as_float(words[i] << 16), v[2 * i + 1] = __uint_as_float(words[i] & 0xffff0000u);
}
__device__ __forceinline__ void store_columns(float* target, const float (&v)[kMixColumns]) {
    reinterpret_cast<float4*>(target)[0] = make_float4(v[0], v[1], v[2], v[3]);
    reinterpret_cast<float4*>(target)[1] = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void store_columns(bf16* target, const float (&v)[kMixColumns]) {
    uint32_t words[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const __nv_bfloat162 pair = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
        words[i] = *reinterpret_cast<const uint32_t*>(&pair);
    }
    *reinterpret_cast<uint4*>(target) = make_uint4(words[0], words[1], words[2], words[3]);
}

// grid: tokens; block kWarps * 32.  projected row: [heads * dim | kv_heads * dim | kv_heads * vdim] from its first column on.
// Dynamic shared memory: rotary / 2 float2 (cosine, sine).
template <typename T>
__global__ void __launch_bounds__(kWarps * 32)
masked_prepare_kernel(const T* __restrict__ projected, long long projected_stride, const float* __restrict__ q_weight, const float* __restrict__ k_weight,
                      float eps, const float* __restrict__ frequency, int rotary, float magnitude, T* __restrict__ queries, T* __restrict__ rows,
                      T* __restrict__ value_pages, const int* __restrict__ positions, const int* __restrict__ token_seq, const int* __restrict__ page_rows, int page_stride,
                      int page_tokens, int heads, int kv_heads, int dim, int vdim, int write_rows, float temperature_coef, int temperature_every,
                      const float* __restrict__ talk, const T* __restrict__ first_values, long long first_stride, const float* __restrict__ value_share) {
    grid_dependents_launch();
    grid_dependency_wait();
    extern __shared__ __align__(16) float2 turns[];       // then, on the next 16-byte border, with `talk`, heads * dim floats: the turned queries
    __shared__ float scratch[33];
    const int token = blockIdx.x;
    const int position = positions[token];
    const int half = rotary / 2;
    for (int pair = threadIdx.x; pair < half; pair += blockDim.x) {
        float sine, cosine;
        sincosf(static_cast<float>(position) * frequency[pair], &sine, &cosine);
        turns[pair] = make_float2(cosine * magnitude, sine * magnitude);
    }
    const T* source = projected + static_cast<size_t>(token) * projected_stride;
    const int q_width = heads * dim, k_width = kv_heads * dim;
    float q_inverse = 1.0f, k_inverse = 1.0f;
    if (q_weight) {
        float squares = 0.0f;
        for (int column = threadIdx.x; column < q_width; column += blockDim.x) {
            const float value = to_float(source[column]);
            squares = fmaf(value, value, squares);
        }
        q_inverse = 1.0f / sqrtf(block_sum(squares, scratch) / static_cast<float>(q_width) + eps);
    }
    if (k_weight && write_rows) {
        float squares = 0.0f;
        for (int column = threadIdx.x; column < k_width; column += blockDim.x) {
            const float value = to_float(source[q_width + column]);
            squares = fmaf(value, value, squares);
        }
        k_inverse = 1.0f / sqrtf(block_sum(squares, scratch) / static_cast<float>(k_width) + eps);
    }
    if (temperature_every > 0) q_inverse *= 1.0f + temperature_coef * logf(static_cast<float>((position + 1) / temperature_every + 1));
    __syncthreads();      // the turns are complete
    // Where the token's keys and values go: head `g`'s key at row + g * key_head_stride, its value at value_row + g * value_head_stride.
    T* row = nullptr;
    T* value_row = nullptr;
    size_t key_head_stride = dim, value_head_stride = vdim;
    if (write_rows) {
        const size_t page = page_rows[static_cast<size_t>(token_seq[token]) * page_stride + position / page_tokens];
        const int within_page = position % page_tokens;
        if (value_pages) {      // keys and values in pages of their own, [pages, kv_heads, page_tokens, dim or vdim]
            key_head_stride = static_cast<size_t>(page_tokens) * dim, value_head_stride = static_cast<size_t>(page_tokens) * vdim;
            row = rows + page * kv_heads * key_head_stride + static_cast<size_t>(within_page) * dim;
            value_row = value_pages + page * kv_heads * value_head_stride + static_cast<size_t>(within_page) * vdim;
        } else {
            row = rows + (page * page_tokens + within_page) * (static_cast<size_t>(kv_heads) * (dim + vdim));
            value_row = row + k_width;
        }
    }
    // Rows that start on 16 bytes, pairs and heads in multiples of 8 elements, no norm weights: a thread takes 8 pairs, or 8 elements that
    // pass, or 8 values at a time.
    float* turned = reinterpret_cast<float*>(turns + (half + 1) / 2 * 2);
    const T* first_row = (write_rows && first_values) ? first_values + static_cast<size_t>(token) * first_stride : nullptr;
    const float share = first_row ? *value_share : 0.0f;
    constexpr uintptr_t kBytes = kMixColumns * sizeof(T) < 16 ? kMixColumns * sizeof(T) - 1 : 15;
    const bool vectors = dim % kMixColumns == 0 && half % kMixColumns == 0 && vdim % kMixColumns == 0 && !q_weight && !k_weight &&
                         ((reinterpret_cast<uintptr_t>(source) | reinterpret_cast<uintptr_t>(queries) | reinterpret_cast<uintptr_t>(row) | reinterpret_cast<uintptr_t>(value_row) |
                           reinterpret_cast<uintptr_t>(first_row)) & kBytes) == 0;
    if (vectors) {
        const int pair_pieces = half / kMixColumns, per_head = dim / kMixColumns - pair_pieces;      // of a head: pieces of pairs, then pieces that pass
        const int head_items = (heads + (write_rows ? kv_heads : 0)) * per_head, value_pieces = vdim / kMixColumns;
        const int all_items = head_items + (write_rows ? kv_heads * value_pieces : 0);
        for (int item = threadIdx.x; item < all_items; item += blockDim.x) {
            float u[kMixColumns];
            if (item >= head_items) {
                const int index = item - head_items, head = index / value_pieces, column = (index - head * value_pieces) * kMixColumns;
                load_columns(source + q_width + k_width + index * kMixColumns, u);
                if (first_row) {
                    float first[kMixColumns];
                    load_columns(first_row + index * kMixColumns, first);
#pragma unroll
                    for (int e = 0; e < kMixColumns; ++e) u[e] = (1.0f - share) * u[e] + share * first[e];
                }
                store_columns(value_row + head * value_head_stride + column, u);
                continue;
            }
            const int any_head = item / per_head, piece = item - any_head * per_head;
            const bool is_query = any_head < heads, pairs = piece < pair_pieces, mix = talk && is_query;
            const int head = is_query ? any_head : any_head - heads, column = pairs ? piece * kMixColumns : half + piece * kMixColumns;
            const float factor = is_query ? q_inverse : 1.0f;
            const T* from = source + (is_query ? 0 : q_width) + head * dim + column;
            T* target = is_query ? queries + static_cast<size_t>(token) * q_width + head * dim + column : row + head * key_head_stride + column;
            float* kept = turned + head * dim + column;
            load_columns(from, u);
#pragma unroll
            for (int e = 0; e < kMixColumns; ++e) u[e] *= factor;
            if (pairs) {
                float w[kMixColumns];
                load_columns(from + half, w);
#pragma unroll
                for (int e = 0; e < kMixColumns; ++e) {
                    const float2 turn = turns[column + e];
                    const float a = u[e], b = w[e] * factor;
                    u[e] = a * turn.x - b * turn.y;
                    w[e] = b * turn.x + a * turn.y;
                }
                if (mix) store_columns(kept + half, w);
                else store_columns(target + half, w);
            }
            if (mix) store_columns(kept, u);
            else store_columns(target, u);
        }
    } else {
        // Within each head, the `half` rotated pairs, then the dim - rotary elements that pass.
        const int per_head = half + (dim - rotary);
        const int all_heads = heads + (write_rows ? kv_heads : 0), lane = threadIdx.x & 31;
        for (int row_head = threadIdx.x >> 5; row_head < all_heads; row_head += kWarps) {      // a warp per head
            const bool is_query = row_head < heads;
            const int head = is_query ? row_head : row_head - heads;
            const T* from = source + (is_query ? 0 : q_width) + head * dim;
            const float* weight = is_query ? q_weight : k_weight;
            const float inverse = is_query ? q_inverse : k_inverse;
            T* target = is_query ? queries + static_cast<size_t>(token) * q_width + head * dim : row + head * key_head_stride;
            for (int within = lane; within < per_head; within += 32) {
                if (within < half) {
                    const int first = within, second = within + half;
                    float u = to_float(from[first]) * inverse, w = to_float(from[second]) * inverse;
                    if (weight) {
                        u *= weight[head * dim + first];
                        w *= weight[head * dim + second];
                    }
                    const float2 turn = turns[within];
                    const float a = u * turn.x - w * turn.y, b = w * turn.x + u * turn.y;
                    if (talk && is_query) {
                        turned[head * dim + first] = a;
                        turned[head * dim + second] = b;
                    } else {
                        target[first] = from_float<T>(a);
                        target[second] = from_float<T>(b);
                    }
                } else {
                    const int column = rotary + (within - half);
                    float u = to_float(from[column]) * inverse;
                    if (weight) u *= weight[head * dim + column];
                    if (talk && is_query) turned[head * dim + column] = u;
                    else target[column] = from_float<T>(u);
                }
            }
        }
        if (write_rows) {
            const T* values = source + q_width + k_width;
            for (int column = threadIdx.x; column < kv_heads * vdim; column += blockDim.x) {
                T value = values[column];
                if (first_row) value = from_float<T>((1.0f - share) * to_float(value) + share * to_float(first_row[column]));
                value_row[(column / vdim) * value_head_stride + column % vdim] = value;
            }
        }
    }
    if (talk) {      // head h's query for key head j: the queries of j's group, weighed by row h of `talk`; rounded once
        __syncthreads();
        const int group_size = heads / kv_heads, wide = kv_heads * dim;
        T* mixed = queries + static_cast<size_t>(token) * heads * wide;
        if (dim % kMixColumns == 0) {
            // A thread takes 8 columns of one key head for a share of the heads, kMixHeads of them at a time.
            const int pieces = wide / kMixColumns, shares = max(1, static_cast<int>(blockDim.x) / pieces);
            for (int item = threadIdx.x; item < pieces * shares; item += blockDim.x) {
                const int piece = item % pieces, group = piece * kMixColumns / dim, column = piece * kMixColumns - group * dim;
                const float* from = turned + group * group_size * dim + column;
                for (int head = item / pieces * kMixHeads; head < heads; head += shares * kMixHeads) {
                    const float* rows_of_talk[kMixHeads];
                    float sum[kMixHeads][kMixColumns];
#pragma unroll
                    for (int i = 0; i < kMixHeads; ++i) {
                        rows_of_talk[i] = talk + (head + i < heads ? head + i : head) * heads + group * group_size;
#pragma unroll
                        for (int e = 0; e < kMixColumns; ++e) sum[i][e] = 0.0f;
                    }
                    for (int g = 0; g < group_size; ++g) {
                        float x[kMixColumns];
                        load_columns(from + g * dim, x);
#pragma unroll
                        for (int i = 0; i < kMixHeads; ++i) {
                            const float weight = rows_of_talk[i][g];
#pragma unroll
                            for (int e = 0; e < kMixColumns; ++e) sum[i][e] = fmaf(weight, x[e], sum[i][e]);
                        }
                    }
#pragma unroll
                    for (int i = 0; i < kMixHeads; ++i)
                        if (head + i < heads) store_columns(mixed + static_cast<size_t>(head + i) * wide + piece * kMixColumns, sum[i]);
                }
            }
            return;
        }
        for (int index = threadIdx.x; index < heads * wide; index += blockDim.x) {
            const int head = index / wide, within = index % wide, group = within / dim, column = within % dim;
            const float* from = turned + group * group_size * dim + column;
            const float* weight = talk + head * heads + group * group_size;
            float sum = 0.0f;
            for (int g = 0; g < group_size; ++g) sum = fmaf(weight[g], from[g * dim], sum);
            mixed[index] = from_float<T>(sum);
        }
    }
}

// grid: (tokens, ceil(heads / kWarps)); a warp per head.  Dynamic shared memory: kWarps * dim floats (the queries).
template <typename T>
__global__ void __launch_bounds__(kWarps * 32)
masked_attention_kernel(const T* __restrict__ queries, const T* __restrict__ rows, const T* __restrict__ value_pages, T* __restrict__ out, long long out_stride,
                        const int* __restrict__ positions, const int* __restrict__ token_seq, const int* __restrict__ page_rows, int page_stride,
                        int page_tokens, int heads, int kv_heads, int dim, int vdim, float scale, int window, int chunk, int sink, float out_scale,
                        const float* __restrict__ distance, int sigmoid_weights, const float* __restrict__ head_offset, const T* __restrict__ gate,
                        long long gate_stride, int gate_per_head, int keep_first, int shared_keys) {
    grid_dependents_launch();
    grid_dependency_wait();
    extern __shared__ float shared[];
    const int token = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int head = blockIdx.y * kWarps + warp;
    if (head >= heads) return;
    // With `shared_keys` a query is `segments` pieces of `dim` elements, one for each key head of the position.
    const int segments = shared_keys ? kv_heads : 1, query_width = segments * dim;
    float* query = shared + static_cast<size_t>(warp) * query_width;
    const T* q_source = queries + (static_cast<size_t>(token) * heads + head) * query_width;
    for (int column = lane; column < query_width; column += 32) query[column] = to_float(q_source[column]) * scale;
    __syncwarp();
    const int position = positions[token];
    const int* pages = page_rows + static_cast<size_t>(token_seq[token]) * page_stride;
    const int group = head / (heads / kv_heads);
    // Position `r` of page `p`: this head's key at keys + p * key_page + r * key_row, its value at values + p * value_page + r * value_row.
    const T* keys;
    const T* values;
    long long key_page, key_row, value_page, value_row;
    const int key_group = shared_keys ? 0 : group;
    const long long key_segment = value_pages ? static_cast<long long>(page_tokens) * dim : dim;      // from one key head's key to the next one's
    if (value_pages) {      // [pages, kv_heads, page_tokens, dim or vdim]
        key_row = dim, value_row = vdim, key_page = static_cast<long long>(kv_heads) * page_tokens * dim, value_page = static_cast<long long>(kv_heads) * page_tokens * vdim;
        keys = rows + static_cast<long long>(key_group) * page_tokens * dim, values = value_pages + static_cast<long long>(group) * page_tokens * vdim;
    } else {                // [pages, page_tokens, keys of all heads | values of all heads]
        key_row = value_row = kv_heads * (dim + vdim), key_page = value_page = key_row * page_tokens;
        keys = rows + key_group * dim, values = rows + kv_heads * dim + group * vdim;
    }
    const Visible seen = visible_keys(position, window, chunk, keep_first);
    float top = sink ? 0.0f : -INFINITY, sum = sink ? 1.0f : 0.0f;       // the sink: a weight of exp(0 - top) that carries no value
    const float far = distance ? distance[2 * head] : 0.0f, reach = distance ? distance[2 * head + 1] : 0.0f;
    const float offset = head_offset ? head_offset[head] : 0.0f;
    float acc[kMaxOwned];
#pragma unroll
    for (int i = 0; i < kMaxOwned; ++i) acc[i] = 0.0f;
    for (int base = 0; base < seen.count; base += 32) {
        const bool valid = base + lane < seen.count;
        const int key = seen.key(base + lane);
        long long value_index = 0;
        float score = -INFINITY;
        if (valid) {
            const long long page = pages[key / page_tokens], within_page = key % page_tokens;
            value_index = page * value_page + within_page * value_row;
            const T* k = keys + page * key_page + within_page * key_row;
            float a = 0.0f, b = 0.0f;
            for (int segment = 0; segment < segments; ++segment, k += key_segment) {
                const float* part = query + segment * dim;
                int column = 0;
                for (; column + 1 < dim; column += 2) {
                    a = fmaf(part[column], to_float(k[column]), a);
                    b = fmaf(part[column + 1], to_float(k[column + 1]), b);
                }
                if (column < dim) a = fmaf(part[column], to_float(k[column]), a);
            }
            score = a + b;
            if (distance) score -= far * log1pf(reach * static_cast<float>(position - key));
        }
        float p;
        if (sigmoid_weights) {
            p = valid ? 1.0f / (1.0f + expf(-(score + offset))) : 0.0f;
        } else {
            const float new_top = fmaxf(top, warp_max(score));       // finite: the block holds at least one key
            p = valid ? expf(score - new_top) : 0.0f;
            const float keep = expf(top - new_top);                   // exp(-inf) = 0 the first time without a sink
            sum = sum * keep + warp_sum(p);
            top = new_top;
#pragma unroll
            for (int i = 0; i < kMaxOwned; ++i) acc[i] *= keep;
        }
        const int count = seen.count - base < 32 ? seen.count - base : 32;
        for (int j = 0; j < count; ++j) {
            const float w = __shfl_sync(0xffffffffu, p, j);
            const T* v = values + __shfl_sync(0xffffffffu, value_index, j);
#pragma unroll
            for (int i = 0; i < kMaxOwned; ++i) {
                const int column = lane + 32 * i;
                if (column < vdim) acc[i] = fmaf(w, to_float(v[column]), acc[i]);
            }
        }
    }
    const float factor = sigmoid_weights ? out_scale : out_scale / sum;
    const T* gates = gate ? gate + static_cast<size_t>(token) * gate_stride + (gate_per_head ? head : head * vdim) : nullptr;
#pragma unroll
    for (int i = 0; i < kMaxOwned; ++i) {
        const int column = lane + 32 * i;
        if (column < vdim) {
            float value = acc[i] * factor;
            if (gates) value /= 1.0f + expf(-to_float(gates[gate_per_head ? 0 : column]));
            out[static_cast<size_t>(token) * out_stride + head * vdim + column] = from_float<T>(value);
        }
    }
}

// ---- single tokens (and any step whose sizes allow): tiles of keys and values staged in shared memory --------------------------
//
// grid: (tokens, kv_heads * ceil(group / kStagedWarps)); block: kStagedWarps warps, one per query head of the key/value head's group.
// All threads bring tiles of 32 positions into shared memory with cp.async, 4 bytes at a time (rows of the cache lie 4-byte
// aligned because dim and vdim are multiples of a word's elements), two tiles deep, so that the group's heads share one pass over
// the cache and the loads are whole rows.  Key rows are an odd number of words apart: lane j reads key j without bank conflicts.
// Then as above: a lane scores one key, every lane sums its own value columns; maximum, weights and sums in 32-bit.
// With `splits` > 1 the grid's z cuts a token's tiles into that many ranges, a block leaves its range's sums, maximum and denominator
// in `partial` ([tokens, heads, splits, vdim + 2] floats), and `masked_attention_merge_kernel` joins them: few tokens over a long
// context then fill the machine.
constexpr int kStagedWarps = 4;
constexpr int kTileKeys = 32;
constexpr int kMaxSplits = 64;

__device__ __forceinline__ void copy_word(void* target, const void* source) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(target))), "l"(source) : "memory");
}
__device__ __forceinline__ void copy_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void copy_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

template <typename T> struct Word;
template <> struct Word<float> {
    static constexpr int kElements = 1;
    static __device__ __forceinline__ float first(uint32_t word) { return __uint_as_float(word); }
    static __device__ __forceinline__ float second(uint32_t) { return 0.0f; }
};
template <> struct Word<bf16> {
    static constexpr int kElements = 2;
    static __device__ __forceinline__ float first(uint32_t word) { return __uint_as_float(word << 16); }
    static __device__ __forceinline__ float second(uint32_t word) { return __uint_as_float(word & 0xffff0000u); }
};

__host__ __device__ inline int key_stride_words(int key_words) { return key_words | 1; }

template <typename T>
__global__ void __launch_bounds__(kStagedWarps * 32)
masked_attention_staged_kernel(const T* __restrict__ queries, const T* __restrict__ rows, const T* __restrict__ value_pages, T* __restrict__ out,
                               long long out_stride, const int* __restrict__ positions, const int* __restrict__ token_seq, const int* __restrict__ page_rows,
                               int page_stride, int page_tokens, int heads, int kv_heads, int dim, int vdim, float scale, int window, int chunk, int sink,
                               float out_scale, const float* __restrict__ distance, int sigmoid_weights, const float* __restrict__ head_offset,
                               const T* __restrict__ gate, long long gate_stride, int gate_per_head, int splits, float* __restrict__ partial, int keep_first) {
    grid_dependents_launch();
    grid_dependency_wait();
    constexpr int kPer = Word<T>::kElements;
    extern __shared__ __align__(16) uint32_t staged_words[];
    const int key_words = dim / kPer, value_words = vdim / kPer, key_stride = key_stride_words(key_words);
    const int tile_words = kTileKeys * (key_stride + value_words);
    float* query_rows = reinterpret_cast<float*>(staged_words + 2 * tile_words);       // [kStagedWarps][dim]
    const int token = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int group_size = heads / kv_heads, passes = (group_size + kStagedWarps - 1) / kStagedWarps;
    const int group = blockIdx.y / passes, head_in_group = (blockIdx.y % passes) * kStagedWarps + warp;
    const bool has_head = head_in_group < group_size;
    const int head = group * group_size + (has_head ? head_in_group : 0);
    const int position = positions[token];
    const int* pages = page_rows + static_cast<size_t>(token_seq[token]) * page_stride;
    const T* keys;
    const T* values;
    long long key_page, key_row, value_page, value_row;
    if (value_pages) {
        key_row = dim, value_row = vdim, key_page = static_cast<long long>(kv_heads) * page_tokens * dim, value_page = static_cast<long long>(kv_heads) * page_tokens * vdim;
        keys = rows + static_cast<long long>(group) * page_tokens * dim, values = value_pages + static_cast<long long>(group) * page_tokens * vdim;
    } else {
        key_row = value_row = kv_heads * (dim + vdim), key_page = value_page = key_row * page_tokens;
        keys = rows + group * dim, values = rows + kv_heads * dim + group * vdim;
    }
    const Visible seen = visible_keys(position, window, chunk, keep_first);
    const int all_tiles = (seen.count - 1) / kTileKeys + 1;
    // This block's range of the token's tiles (all of them without splits); tiles are numbered from the range's first.
    const int per_split = (all_tiles + splits - 1) / splits, tile_begin = static_cast<int>(blockIdx.z) * per_split;
    const int n_tiles = all_tiles - tile_begin < per_split ? (all_tiles - tile_begin > 0 ? all_tiles - tile_begin : 0) : per_split;
    const int first_number = tile_begin * kTileKeys;      // of the range's first tile, among the keys that the token sees

    auto stage = [&](int tile) {
        uint32_t* buffer = staged_words + (tile & 1) * tile_words;
        if (tile < n_tiles) {
            const int base = first_number + tile * kTileKeys;
            const int count = seen.count - base < kTileKeys ? seen.count - base : kTileKeys;
            uint32_t* value_buffer = buffer + kTileKeys * key_stride;
            for (int row = warp; row < count; row += kStagedWarps) {      // a warp per row: one page lookup, then whole lines
                const int key = seen.key(base + row);
                const long long page = pages[key / page_tokens], within_page = key % page_tokens;
                const uint32_t* key_source = reinterpret_cast<const uint32_t*>(keys + page * key_page + within_page * key_row);
                const uint32_t* value_source = reinterpret_cast<const uint32_t*>(values + page * value_page + within_page * value_row);
                for (int word = lane; word < key_words; word += 32) copy_word(buffer + row * key_stride + word, key_source + word);
                for (int word = lane; word < value_words; word += 32) copy_word(value_buffer + row * value_words + word, value_source + word);
            }
        }
        copy_commit();
    };
    stage(0);
    stage(1);
    if (has_head)
        for (int column = lane; column < dim; column += 32)
            query_rows[warp * dim + column] = to_float(queries[(static_cast<size_t>(token) * heads + head) * dim + column]) * scale;
    const float* query = query_rows + warp * dim;
    const float far = distance ? distance[2 * head] : 0.0f, reach = distance ? distance[2 * head + 1] : 0.0f;
    const float offset = head_offset ? head_offset[head] : 0.0f;
    const bool with_sink = sink && blockIdx.z == 0;      // the added one is counted once
    float top = with_sink ? 0.0f : -INFINITY, sum = with_sink ? 1.0f : 0.0f;
    float acc[kMaxOwned];
#pragma unroll
    for (int i = 0; i < kMaxOwned; ++i) acc[i] = 0.0f;
    for (int tile = 0; tile < n_tiles; ++tile) {
        copy_wait<1>();      // this thread's copies of `tile` are done (those of the next tile may be on their way)
        __syncthreads();     // everybody's are; the queries too
        const uint32_t* buffer = staged_words + (tile & 1) * tile_words;
        const int base = first_number + tile * kTileKeys;
        const int count = seen.count - base < kTileKeys ? seen.count - base : kTileKeys;
        if (has_head) {
            float score = -INFINITY;
            if (lane < count) {
                const uint32_t* k = buffer + lane * key_stride;
                float a = 0.0f, b = 0.0f;
                for (int word = 0; word < key_words; ++word) {
                    const uint32_t both = k[word];
                    a = fmaf(query[word * kPer], Word<T>::first(both), a);
                    if (kPer == 2) b = fmaf(query[word * kPer + 1], Word<T>::second(both), b);
                }
                score = a + b;
                if (distance) score -= far * log1pf(reach * static_cast<float>(position - seen.key(base + lane)));
            }
            float p;
            if (sigmoid_weights) {
                p = lane < count ? 1.0f / (1.0f + expf(-(score + offset))) : 0.0f;
            } else {
                const float new_top = fmaxf(top, warp_max(score));
                p = lane < count ? expf(score - new_top) : 0.0f;
                const float keep = expf(top - new_top);
                sum = sum * keep + warp_sum(p);
                top = new_top;
#pragma unroll
                for (int i = 0; i < kMaxOwned; ++i) acc[i] *= keep;
            }
            const uint32_t* v = buffer + kTileKeys * key_stride;
            for (int j = 0; j < count; ++j) {
                const float w = __shfl_sync(0xffffffffu, p, j);
#pragma unroll
                for (int i = 0; i < kMaxOwned / kPer; ++i) {
                    const int word = lane + 32 * i;
                    if (word < value_words) {
                        const uint32_t both = v[j * value_words + word];
                        acc[i * kPer] = fmaf(w, Word<T>::first(both), acc[i * kPer]);
                        if (kPer == 2) acc[i * kPer + 1] = fmaf(w, Word<T>::second(both), acc[i * kPer + 1]);
                    }
                }
            }
        }
        __syncthreads();     // the tile's place may be written over
        stage(tile + 2);
    }
    copy_wait<0>();
    if (!has_head) return;
    if (partial) {      // this range's sums as they stand (in the scale of its own maximum), then the maximum and the denominator
        float* record = partial + ((static_cast<size_t>(token) * heads + head) * splits + blockIdx.z) * (vdim + 2);
#pragma unroll
        for (int i = 0; i < kMaxOwned / kPer; ++i) {
            const int word = lane + 32 * i;
            if (word < value_words) {
#pragma unroll
                for (int e = 0; e < kPer; ++e) record[word * kPer + e] = acc[i * kPer + e];
            }
        }
        if (lane == 0) record[vdim] = top, record[vdim + 1] = sum;
        return;
    }
    const float factor = sigmoid_weights ? out_scale : out_scale / sum;
    T* target = out + static_cast<size_t>(token) * out_stride + head * vdim;
    const T* gates = gate ? gate + static_cast<size_t>(token) * gate_stride + (gate_per_head ? head : head * vdim) : nullptr;
#pragma unroll
    for (int i = 0; i < kMaxOwned / kPer; ++i) {
        const int word = lane + 32 * i;
        if (word < value_words) {
#pragma unroll
            for (int e = 0; e < kPer; ++e) {
                float value = acc[i * kPer + e] * factor;
                if (gates) value /= 1.0f + expf(-to_float(gates[gate_per_head ? 0 : word * kPer + e]));
                target[word * kPer + e] = from_float<T>(value);
            }
        }
    }
}

// grid (tokens, heads); block 128.  Joins the ranges that the staged kernel left in `partial`: the sums are brought to the largest
// maximum and added, divided by the joined denominator (sigmoid weights: added as they are), gated and rounded once.
template <typename T>
__global__ void __launch_bounds__(128)
masked_attention_merge_kernel(const float* __restrict__ partial, T* __restrict__ out, long long out_stride, int heads, int vdim, int splits, float out_scale,
                              int sigmoid_weights, const T* __restrict__ gate, long long gate_stride, int gate_per_head) {
    grid_dependents_launch();
    grid_dependency_wait();
    __shared__ float factors[kMaxSplits];
    const int token = blockIdx.x, head = blockIdx.y;
    const float* records = partial + (static_cast<size_t>(token) * heads + head) * splits * (vdim + 2);
    // The first warp turns the ranges' maxima and denominators into the factors of their sums.
    if (threadIdx.x < 32) {
        float tops[kMaxSplits / 32], top = -INFINITY, total = 0.0f;
#pragma unroll
        for (int i = 0; i < kMaxSplits / 32; ++i) {
            const int split = threadIdx.x + 32 * i;
            tops[i] = (!sigmoid_weights && split < splits) ? records[static_cast<size_t>(split) * (vdim + 2) + vdim] : -INFINITY;
            top = fmaxf(top, tops[i]);
        }
        top = warp_max(top);
#pragma unroll
        for (int i = 0; i < kMaxSplits / 32; ++i) {
            const int split = threadIdx.x + 32 * i;
            tops[i] = expf(tops[i] - top);                       // a range without keys: exp(-inf) = 0
            if (!sigmoid_weights && split < splits) total = fmaf(records[static_cast<size_t>(split) * (vdim + 2) + vdim + 1], tops[i], total);
        }
        total = warp_sum(total);
#pragma unroll
        for (int i = 0; i < kMaxSplits / 32; ++i) factors[threadIdx.x + 32 * i] = sigmoid_weights ? out_scale : tops[i] * (out_scale / total);
    }
    __syncthreads();
    const T* gates = gate ? gate + static_cast<size_t>(token) * gate_stride + (gate_per_head ? head : head * vdim) : nullptr;
    for (int column = threadIdx.x; column < vdim; column += blockDim.x) {
        float sum = 0.0f;
#pragma unroll 8
        for (int split = 0; split < splits; ++split) sum = fmaf(records[static_cast<size_t>(split) * (vdim + 2) + column], factors[split], sum);
        if (gates) sum /= 1.0f + expf(-to_float(gates[gate_per_head ? 0 : column]));
        out[static_cast<size_t>(token) * out_stride + head * vdim + column] = from_float<T>(sum);
    }
}

// ---- single tokens with mixed scores ---------------------------------------------------------------------------------------------
//
// grid: (tokens, splits); block: kTalkWarps warps that serve all heads of a token together, since every head's weights need every head's
// scores.  Tiles of 32 positions, keys and values of all key/value heads, come into shared memory by cp.async, 16 bytes at a time (one or
// two tiles deep, as they fit); key rows are an odd number of 16-byte units apart.  Then, for each tile:
//   scores    lane = key; a warp takes two heads of one key head at a time, so that a key's elements are read once for both;
//   mixing    lane = key; a warp takes a head: sum over all heads of talk[h, g] * score_g, running maximum, weights and sum;
//   values    a thread owns 16 bytes' worth of a head's columns (kOwned such places) and adds the tile's weighted values to them.
// Scores, mixing, weights and sums in 32-bit.  `splits` > 1: ranges joined by `masked_attention_merge_kernel`, as above.
constexpr int kTalkWarps = 8;
constexpr int kScoreStride = kTileKeys + 1;

__device__ __forceinline__ void copy_16(void* target, const void* source) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(target))), "l"(source) : "memory");
}

// The elements of 16 bytes as floats.
__device__ __forceinline__ void unpack_16(uint4 raw, float (&v)[8], bf16) {
    const uint32_t words[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) v[2 * i] = __uint_as_float(words[i] << 16), v[2 * i + 1] = __uint_as_float(words[i] & 0xffff0000u);
}
__device__ __forceinline__ void unpack_16(uint4 raw, float (&v)[4], float) {
    v[0] = __uint_as_float(raw.x), v[1] = __uint_as_float(raw.y), v[2] = __uint_as_float(raw.z), v[3] = __uint_as_float(raw.w);
}

// Shared memory by section, in bytes.
struct TalkPlan {
    int key_stride, value_stride, tile, stages, total;      // of a staged row of keys and of values, of one tile, tiles in flight, all together
};
template <typename T>
__host__ __device__ inline TalkPlan talk_plan(int heads, int kv_heads, int dim, int vdim) {
    TalkPlan plan = {0, 0, 0, 0, 0};
    constexpr int kPer = 16 / static_cast<int>(sizeof(T));
    if (dim % kPer != 0 || vdim % kPer != 0) return plan;
    plan.key_stride = ((kv_heads * dim / kPer) | 1) * 16;
    plan.value_stride = kv_heads * vdim / kPer * 16;
    const long long tile = static_cast<long long>(kTileKeys) * (plan.key_stride + plan.value_stride);
    const long long fixed = 4LL * (static_cast<long long>(heads) * dim + heads * heads + 2LL * heads * kScoreStride + 3LL * heads);
    if (tile + fixed > kMaxShared) return plan;
    plan.tile = static_cast<int>(tile);
    plan.stages = 2 * tile + fixed <= kMaxShared ? 2 : 1;
    plan.total = static_cast<int>(plan.stages * tile + fixed);
    return plan;
}

template <typename T, int kOwned>
__global__ void __launch_bounds__(kTalkWarps * 32)
talking_decode_kernel(const T* __restrict__ queries, const T* __restrict__ rows, const T* __restrict__ value_pages, const float* __restrict__ talk,
                      T* __restrict__ out, long long out_stride, const int* __restrict__ positions, const int* __restrict__ token_seq,
                      const int* __restrict__ page_rows, int page_stride, int page_tokens, int heads, int kv_heads, int dim, int vdim, float scale, int window,
                      int keep_first, float out_scale, int splits, float* __restrict__ partial) {
    grid_dependents_launch();
    constexpr int kPer = 16 / static_cast<int>(sizeof(T)), kThreads = kTalkWarps * 32;
    extern __shared__ __align__(16) uint8_t talk_shared[];
    const TalkPlan plan = talk_plan<T>(heads, kv_heads, dim, vdim);
    float* query = reinterpret_cast<float*>(talk_shared + plan.stages * plan.tile);      // [heads][dim], scaled
    float* mixing = query + heads * dim;                                                  // [heads][heads]
    float* scores = mixing + heads * heads;                                               // [heads][kScoreStride]
    float* weights = scores + heads * kScoreStride;                                       // the same
    float* tops = weights + heads * kScoreStride;                                         // [heads] running maxima, sums, and the last rescaling
    float* sums = tops + heads;
    float* rescale = sums + heads;
    const int token = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int index = threadIdx.x; index < heads * heads; index += kThreads) mixing[index] = talk[index];      // a weight: no earlier kernel writes it
    for (int head = threadIdx.x; head < heads; head += kThreads) tops[head] = -INFINITY, sums[head] = 0.0f;
    grid_dependency_wait();
    const int position = positions[token];
    const int* pages = page_rows + static_cast<size_t>(token_seq[token]) * page_stride;
    const Visible seen = visible_keys(position, window, 0, keep_first);
    const int all_tiles = (seen.count - 1) / kTileKeys + 1;
    const int per_split = (all_tiles + splits - 1) / splits, tile_begin = static_cast<int>(blockIdx.y) * per_split;
    const int n_tiles = all_tiles - tile_begin < per_split ? (all_tiles - tile_begin > 0 ? all_tiles - tile_begin : 0) : per_split;
    const int first_number = tile_begin * kTileKeys;
    const int key_pieces = dim / kPer, value_pieces = vdim / kPer;      // 16-byte pieces of one head's key and value
    const int row_pieces = kv_heads * (key_pieces + value_pieces);
    auto stage = [&](int tile) {
        if (tile < n_tiles) {
            uint8_t* buffer = talk_shared + (plan.stages == 2 ? (tile & 1) * plan.tile : 0);
            const int base = first_number + tile * kTileKeys;
            const int count = seen.count - base < kTileKeys ? seen.count - base : kTileKeys;
            for (int row = warp; row < count; row += kTalkWarps) {      // a warp per row: one page lookup, then whole lines
                const int key = seen.key(base + row);
                const long long page = pages[key / page_tokens], within = key % page_tokens;
                uint8_t* key_target = buffer + row * plan.key_stride;
                uint8_t* value_target = buffer + kTileKeys * plan.key_stride + row * plan.value_stride;
                for (int piece = lane; piece < row_pieces; piece += 32) {
                    const bool is_key = piece < kv_heads * key_pieces;
                    const int index = is_key ? piece : piece - kv_heads * key_pieces;
                    const T* source;
                    if (value_pages) {
                        const int per = is_key ? key_pieces : value_pieces, head = index / per;
                        source = (is_key ? rows : value_pages) + ((page * kv_heads + head) * page_tokens + within) * (is_key ? dim : vdim) + (index - head * per) * kPer;
                    } else {
                        source = rows + (page * page_tokens + within) * (static_cast<long long>(kv_heads) * (dim + vdim)) + piece * kPer;
                    }
                    copy_16((is_key ? key_target : value_target) + index * 16, source);
                }
            }
        }
        copy_commit();
    };
    stage(0);
    if (plan.stages == 2) stage(1);
    for (int index = threadIdx.x; index < heads * dim; index += kThreads) query[index] = to_float(queries[static_cast<size_t>(token) * heads * dim + index]) * scale;
    float acc[kOwned][kPer];
#pragma unroll
    for (int i = 0; i < kOwned; ++i)
#pragma unroll
        for (int e = 0; e < kPer; ++e) acc[i][e] = 0.0f;
    const int group_size = heads / kv_heads, pairs = (group_size + 1) / 2;
    for (int tile = 0; tile < n_tiles; ++tile) {
        if (plan.stages == 2) copy_wait<1>();
        else copy_wait<0>();
        __syncthreads();     // the tile has arrived for everybody; the queries and the mixing weights are there
        const uint8_t* buffer = talk_shared + (plan.stages == 2 ? (tile & 1) * plan.tile : 0);
        const int base = first_number + tile * kTileKeys;
        const int count = seen.count - base < kTileKeys ? seen.count - base : kTileKeys;
        for (int item = warp; item < kv_heads * pairs; item += kTalkWarps) {
            const int group = item / pairs, in_group = item % pairs * 2, head = group * group_size + in_group;
            const bool second = in_group + 1 < group_size;
            if (lane < count) {
                const uint4* k = reinterpret_cast<const uint4*>(buffer + lane * plan.key_stride) + group * key_pieces;
                const float* q0 = query + head * dim;
                const float* q1 = second ? q0 + dim : q0;
                float a[2] = {0.0f, 0.0f}, b[2] = {0.0f, 0.0f};
                for (int piece = 0; piece < key_pieces; ++piece) {
                    float v[kPer];
                    unpack_16(k[piece], v, T());
#pragma unroll
                    for (int e = 0; e < kPer; e += 4) {
                        const float4 x = *reinterpret_cast<const float4*>(q0 + piece * kPer + e), y = *reinterpret_cast<const float4*>(q1 + piece * kPer + e);
                        a[0] = fmaf(x.x, v[e], a[0]), a[1] = fmaf(x.y, v[e + 1], a[1]), a[0] = fmaf(x.z, v[e + 2], a[0]), a[1] = fmaf(x.w, v[e + 3], a[1]);
                        b[0] = fmaf(y.x, v[e], b[0]), b[1] = fmaf(y.y, v[e + 1], b[1]), b[0] = fmaf(y.z, v[e + 2], b[0]), b[1] = fmaf(y.w, v[e + 3], b[1]);
                    }
                }
                scores[head * kScoreStride + lane] = a[0] + a[1];
                if (second) scores[(head + 1) * kScoreStride + lane] = b[0] + b[1];
            }
        }
        __syncthreads();
        for (int head = warp; head < heads; head += kTalkWarps) {
            float mixed = -INFINITY;
            if (lane < count) {
                float sum[2] = {0.0f, 0.0f};
                for (int g = 0; g < heads; ++g) sum[g & 1] = fmaf(mixing[head * heads + g], scores[g * kScoreStride + lane], sum[g & 1]);
                mixed = sum[0] + sum[1];
            }
            const float top = tops[head], new_top = fmaxf(top, warp_max(mixed));
            const float p = lane < count ? expf(mixed - new_top) : 0.0f, total = warp_sum(p);
            weights[head * kScoreStride + lane] = p;
            __syncwarp();      // every lane has read the maximum
            if (lane == 0) {
                const float keep = expf(top - new_top);      // exp(-inf) = 0 the first time
                tops[head] = new_top, sums[head] = sums[head] * keep + total, rescale[head] = keep;
            }
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < kOwned; ++i) {
            const int place = threadIdx.x + i * kThreads;
            if (place < heads * value_pieces) {
                const int head = place / value_pieces, piece = place % value_pieces;
                const float keep = rescale[head];
#pragma unroll
                for (int e = 0; e < kPer; ++e) acc[i][e] *= keep;
                const uint8_t* v = buffer + kTileKeys * plan.key_stride + (head / group_size * value_pieces + piece) * 16;
                const float* weight = weights + head * kScoreStride;
                for (int j = 0; j < count; ++j) {
                    float value[kPer];
                    unpack_16(*reinterpret_cast<const uint4*>(v + j * plan.value_stride), value, T());
                    const float w = weight[j];
#pragma unroll
                    for (int e = 0; e < kPer; ++e) acc[i][e] = fmaf(w, value[e], acc[i][e]);
                }
            }
        }
        __syncthreads();     // the tile's place may be written over
        stage(tile + plan.stages);
    }
    copy_wait<0>();
#pragma unroll
    for (int i = 0; i < kOwned; ++i) {
        const int place = threadIdx.x + i * kThreads;
        if (place >= heads * value_pieces) continue;
        const int head = place / value_pieces, piece = place % value_pieces;
        if (partial) {
            float* record = partial + ((static_cast<size_t>(token) * heads + head) * splits + blockIdx.y) * (vdim + 2);
#pragma unroll
            for (int e = 0; e < kPer; ++e) record[piece * kPer + e] = acc[i][e];
            if (piece == 0) record[vdim] = tops[head], record[vdim + 1] = sums[head];
        } else {
            const float factor = out_scale / sums[head];
            T* target = out + static_cast<size_t>(token) * out_stride + head * vdim + piece * kPer;
#pragma unroll
            for (int e = 0; e < kPer; ++e) target[e] = from_float<T>(acc[i][e] * factor);
        }
    }
}

template <typename T>
bool talk_fits(int heads, int kv_heads, int dim, int vdim) {
    return heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dim > 0 && vdim > 0 && static_cast<long long>(heads) * vdim * sizeof(T) <= 4LL * 16 * kTalkWarps * 32 &&
           talk_plan<T>(heads, kv_heads, dim, vdim).total > 0;
}

template <typename T>
int launch_talking_decode(const void* queries, const void* rows, const void* value_pages, const float* talk, void* out, long long out_stride, const int* positions,
                          const int* token_seq, const int* page_rows, int page_stride, int page_tokens, int tokens, int heads, int kv_heads, int dim, int vdim,
                          float scale, int window, int keep_first, float out_scale, int splits, float* partial, cudaStream_t s) {
    if (!talk_fits<T>(heads, kv_heads, dim, vdim)) return cudaErrorInvalidValue;
    const TalkPlan plan = talk_plan<T>(heads, kv_heads, dim, vdim);
    const int places = heads * vdim * static_cast<int>(sizeof(T)) / 16, owned = (places + kTalkWarps * 32 - 1) / (kTalkWarps * 32);
    if ((splits > 1 && !partial) || splits > kMaxSplits) return cudaErrorInvalidValue;
    if (splits <= 1) splits = 1, partial = nullptr;
#define TAU_TALK(OWNED)                                                                                                                                          \
    {                                                                                                                                                            \
        const cudaError_t status = cudaFuncSetAttribute(talking_decode_kernel<T, OWNED>, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxShared);                \
        if (status != cudaSuccess) return static_cast<int>(status);                                                                                              \
        tau_launch(talking_decode_kernel<T, OWNED>, dim3(tokens, splits), dim3(kTalkWarps * 32), plan.total, s, static_cast<const T*>(queries),                   \
                   static_cast<const T*>(rows), static_cast<const T*>(value_pages), talk, static_cast<T*>(out), out_stride, positions, token_seq, page_rows,       \
                   page_stride, page_tokens, heads, kv_heads, dim, vdim, scale, window, keep_first, out_scale, splits, partial);                                  \
    }
    if (owned <= 1) TAU_TALK(1)
    else if (owned <= 2) TAU_TALK(2)
    else TAU_TALK(4)
#undef TAU_TALK
    const int status = tau_launch_status();
    if (status != 0 || !partial) return status;
    tau_launch(masked_attention_merge_kernel<T>, dim3(tokens, heads), dim3(128), 0, s, partial, static_cast<T*>(out), out_stride, heads, vdim, splits, out_scale, 0,
               static_cast<const T*>(nullptr), 0LL, 0);
    return tau_launch_status();
}

// ---- single tokens in bfloat16 against the keys of all key heads side by side ------------------------------------------------------
//
// The mixed queries of a token (prepare's, one piece for each key head) are a matrix of `heads` rows and kv_heads * dim columns, and every row
// asks the same keys: a product for the tensor cores whose rows are the heads.  grid: (tokens, splits); block: kSharedWarps warps.  A tile is
// kKeys positions, keys and values of all key/value heads, by cp.async (the values' copies run on beside the scores):
//   scores    a warp takes 16 heads and 8 keys: mma.sync m16n8k16 over all key heads' elements, operands by ldmatrix;
//   weights   a warp takes a head: mask, running maximum, weights (rounded to bfloat16 as the second product's operand) and their 32-bit sum;
//   values    an item is 16 heads of one value head's group (rows beyond the group are not kept) and 8 of its columns: mma.sync over the keys.
// Scores, weights and sums in 32-bit; accumulators in registers, kItems items to a warp.  `splits` > 1: joined by `masked_attention_merge_kernel`.
constexpr int kSharedWarps = 8;

struct SharedPlan {
    int keys, items;                                             // positions of a tile, items of a warp; keys = 0: not served
    int head_rows, query_stride, key_stride, value_stride;       // rows of 16-head tiles; bytes of a staged row
    int key_offset, value_offset, score_offset, weight_offset, stat_offset, total;
};
__host__ __device__ inline int odd_units(int bytes) { return ((bytes / 16) | 1) * 16; }      // rows an odd number of 16-byte units apart: no bank conflicts
__host__ __device__ inline SharedPlan shared_plan(int heads, int kv_heads, int dim, int vdim, int keys) {
    SharedPlan plan = {};
    const int wide = kv_heads * dim, group_tiles = (heads / kv_heads + 15) / 16;
    if (dim % 8 != 0 || vdim % 8 != 0 || wide % 32 != 0 || heads > 256) return plan;
    plan.items = (kv_heads * group_tiles * (vdim / 8) + kSharedWarps - 1) / kSharedWarps;
    plan.head_rows = (heads + 15) / 16 * 16;
    plan.query_stride = odd_units(wide * 2), plan.key_stride = plan.query_stride, plan.value_stride = odd_units(kv_heads * vdim * 2);
    const long long query = static_cast<long long>(plan.head_rows) * plan.query_stride, key = static_cast<long long>(keys) * plan.key_stride;
    const long long value = static_cast<long long>(keys) * plan.value_stride, score = static_cast<long long>(plan.head_rows) * (keys + 4) * 4;
    const long long weight = static_cast<long long>(plan.head_rows + 16) * (keys + 8) * 2, total = query + key + value + score + weight + 3LL * plan.head_rows * 4;
    if (total > kMaxShared || plan.items > 16) return plan;
    plan.key_offset = static_cast<int>(query), plan.value_offset = static_cast<int>(query + key), plan.score_offset = static_cast<int>(query + key + value);
    plan.weight_offset = plan.score_offset + static_cast<int>(score), plan.stat_offset = plan.weight_offset + static_cast<int>(weight);
    plan.total = static_cast<int>(total);
    plan.keys = keys;
    return plan;
}

__device__ __forceinline__ void load_matrices(uint32_t (&r)[4], uint32_t address) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(address) : "memory");
}
__device__ __forceinline__ void load_matrices_transposed(uint32_t (&r)[4], uint32_t address) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(address) : "memory");
}
__device__ __forceinline__ void multiply_add(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

template <int kKeys, int kItems>
__global__ void __launch_bounds__(kSharedWarps * 32)
shared_key_decode_kernel(const bf16* __restrict__ queries, const bf16* __restrict__ rows, const bf16* __restrict__ value_pages, bf16* __restrict__ out,
                         long long out_stride, const int* __restrict__ positions, const int* __restrict__ token_seq, const int* __restrict__ page_rows,
                         int page_stride, int page_tokens, int heads, int kv_heads, int dim, int vdim, float scale, int window, int keep_first, float out_scale,
                         int splits, float* __restrict__ partial) {
    grid_dependents_launch();
    constexpr int kThreads = kSharedWarps * 32, kScoreStride = kKeys + 4, kWeightStride = kKeys + 8;
    extern __shared__ __align__(16) uint8_t shared_bytes[];
    const SharedPlan plan = shared_plan(heads, kv_heads, dim, vdim, kKeys);
    float* scores = reinterpret_cast<float*>(shared_bytes + plan.score_offset);        // [head_rows][kScoreStride]
    bf16* weights = reinterpret_cast<bf16*>(shared_bytes + plan.weight_offset);         // [head_rows + 16][kWeightStride]
    float* tops = reinterpret_cast<float*>(shared_bytes + plan.stat_offset);            // running maxima, sums, the last rescaling
    float* sums = tops + plan.head_rows;
    float* rescale = sums + plan.head_rows;
    const uint32_t base = static_cast<uint32_t>(__cvta_generic_to_shared(shared_bytes));
    const int token = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, matrix = lane >> 3, matrix_row = lane & 7;
    const int wide = kv_heads * dim, key_pieces = wide / 8, value_pieces = kv_heads * vdim / 8;      // 16-byte pieces of a position
    for (int head = threadIdx.x; head < plan.head_rows; head += kThreads) tops[head] = -INFINITY, sums[head] = 0.0f, rescale[head] = 0.0f;
    grid_dependency_wait();
    const int position = positions[token];
    const int* pages = page_rows + static_cast<size_t>(token_seq[token]) * page_stride;
    const Visible seen = visible_keys(position, window, 0, keep_first);
    const int all_tiles = (seen.count - 1) / kKeys + 1;
    const int per_split = (all_tiles + splits - 1) / splits, tile_begin = static_cast<int>(blockIdx.y) * per_split;
    const int n_tiles = all_tiles - tile_begin < per_split ? (all_tiles - tile_begin > 0 ? all_tiles - tile_begin : 0) : per_split;
    // Rows of keys or of values of a tile: a warp brings rows warp, warp + kSharedWarps, ...; lane n knows where the n-th of them lies (`place`,
    // in positions of the cache; -1 behind the tile's last one, where zeros go: the weights there are zero, what lies there is not known).
    auto stage = [&](long long place, bool is_key) {
        const int pieces = is_key ? key_pieces : value_pieces, size = is_key ? dim : vdim, per_head = size / 8;
        uint8_t* buffer = shared_bytes + (is_key ? plan.key_offset : plan.value_offset);
        const int stride = is_key ? plan.key_stride : plan.value_stride;
        const bf16* source = value_pages && !is_key ? value_pages : rows + (value_pages || is_key ? 0 : wide);
        const long long row_width = value_pages ? size : static_cast<long long>(wide) + kv_heads * vdim;
        for (int first = 0; first < pieces; first += 32) {
            const int piece = first + lane, head = piece / per_head;
            const bf16* from = source + (value_pages ? static_cast<long long>(head) * page_tokens * size + (piece - head * per_head) * 8 : piece * 8LL);
            uint8_t* target = buffer + warp * stride + piece * 16;
#pragma unroll
            for (int n = 0; n < kKeys / kSharedWarps; ++n) {
                const long long at = __shfl_sync(0xffffffffu, place, n);
                if (piece < pieces) {
                    if (at >= 0) copy_16(target + n * kSharedWarps * stride, from + at * row_width);
                    else *reinterpret_cast<uint4*>(target + n * kSharedWarps * stride) = make_uint4(0u, 0u, 0u, 0u);
                }
            }
        }
        copy_commit();
    };
    // The token's queries, with the first tile's keys.
    for (int head = warp; head < heads; head += kSharedWarps)
        for (int piece = lane; piece < key_pieces; piece += 32)
            copy_16(shared_bytes + head * plan.query_stride + piece * 16, queries + (static_cast<size_t>(token) * heads + head) * wide + piece * 8);
    float acc[kItems][4];
#pragma unroll
    for (int i = 0; i < kItems; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[i][e] = 0.0f;
    const int group_size = heads / kv_heads, group_tiles = (group_size + 15) / 16, columns = vdim / 8, items = kv_heads * group_tiles * columns;
    for (int tile = 0; tile < n_tiles; ++tile) {
        const int base_number = (tile_begin + tile) * kKeys;
        const int count = seen.count - base_number < kKeys ? seen.count - base_number : kKeys;
        const int row = warp + kSharedWarps * lane;
        long long place = -1;
        if (lane < kKeys / kSharedWarps && row < count) {
            const int key = seen.key(base_number + row);
            place = static_cast<long long>(pages[key / page_tokens]) * (value_pages ? kv_heads : 1) * page_tokens + key % page_tokens;
        }
        stage(place, true);
        stage(place, false);
        copy_wait<1>();
        __syncthreads();     // the keys (and the queries) have arrived for everybody
        for (int item = warp; item < plan.head_rows / 16 * (kKeys / 8); item += kSharedWarps) {
            const int head0 = item / (kKeys / 8) * 16, key0 = item % (kKeys / 8) * 8;
            const uint32_t a_address = base + (head0 + matrix_row + (matrix & 1) * 8) * plan.query_stride + (matrix >> 1) * 16;
            const uint32_t b_address = base + plan.key_offset + (key0 + matrix_row) * plan.key_stride + matrix * 16;
            float c[2][4] = {{0.0f, 0.0f, 0.0f, 0.0f}, {0.0f, 0.0f, 0.0f, 0.0f}};
#pragma unroll 4
            for (int k = 0; k < wide; k += 32) {
                uint32_t a0[4], a1[4], b[4];
                load_matrices(b, b_address + k * 2);
                load_matrices(a0, a_address + k * 2);
                load_matrices(a1, a_address + k * 2 + 32);
                multiply_add(c[0], a0, b[0], b[1]);
                multiply_add(c[1], a1, b[2], b[3]);
            }
            float* target = scores + (head0 + (lane >> 2)) * kScoreStride + key0 + (lane & 3) * 2;
            target[0] = c[0][0] + c[1][0], target[1] = c[0][1] + c[1][1];
            target[8 * kScoreStride] = c[0][2] + c[1][2], target[8 * kScoreStride + 1] = c[0][3] + c[1][3];
        }
        __syncthreads();
        for (int head = warp; head < heads; head += kSharedWarps) {
            float value[kKeys / 32], tile_top = -INFINITY, total = 0.0f;
#pragma unroll
            for (int i = 0; i < kKeys / 32; ++i) {
                const int key = lane + 32 * i;
                value[i] = key < count ? scores[head * kScoreStride + key] * scale : -INFINITY;
                tile_top = fmaxf(tile_top, value[i]);
            }
            const float top = tops[head], new_top = fmaxf(top, warp_max(tile_top));
#pragma unroll
            for (int i = 0; i < kKeys / 32; ++i) {
                const float p = expf(value[i] - new_top);      // exp(-inf) = 0 behind the last key
                total += p;
                weights[head * kWeightStride + lane + 32 * i] = __float2bfloat16_rn(p);
            }
            total = warp_sum(total);      // every lane has read the maximum by now
            if (lane == 0) {
                const float keep = expf(top - new_top);
                tops[head] = new_top, sums[head] = sums[head] * keep + total, rescale[head] = keep;
            }
        }
        copy_wait<0>();
        __syncthreads();     // weights and values are there
#pragma unroll
        for (int i = 0; i < kItems; ++i) {
            const int item = warp + i * kSharedWarps;
            if (item < items) {
                const int column = item % columns, group_tile = item / columns, group = group_tile / group_tiles;
                const int head0 = group * group_size + group_tile % group_tiles * 16, end = (group + 1) * group_size;
                const int low = head0 + (lane >> 2), high = low + 8;
                const float keep_low = low < end ? rescale[low] : 0.0f, keep_high = high < end ? rescale[high] : 0.0f;
                acc[i][0] *= keep_low, acc[i][1] *= keep_low, acc[i][2] *= keep_high, acc[i][3] *= keep_high;
                const uint32_t a_address = base + plan.weight_offset + ((head0 + matrix_row + (matrix & 1) * 8) * kWeightStride + (matrix >> 1) * 8) * 2;
                const uint32_t b_address = base + plan.value_offset + lane * plan.value_stride + (group * vdim + column * 8) * 2;
#pragma unroll
                for (int k = 0; k < kKeys; k += 32) {
                    uint32_t a0[4], a1[4], b[4];
                    load_matrices(a0, a_address + k * 2);
                    load_matrices(a1, a_address + k * 2 + 32);
                    load_matrices_transposed(b, b_address + k * plan.value_stride);
                    multiply_add(acc[i], a0, b[0], b[1]);
                    multiply_add(acc[i], a1, b[2], b[3]);
                }
            }
        }
        __syncthreads();     // the tile's place may be written over
    }
    copy_commit();       // (a block whose range is empty has asked for the queries alone)
    copy_wait<0>();
#pragma unroll
    for (int i = 0; i < kItems; ++i) {
        const int item = warp + i * kSharedWarps;
        if (item >= items) continue;
        const int column = item % columns, group_tile = item / columns, group = group_tile / group_tiles;
        const int head0 = group * group_size + group_tile % group_tiles * 16, end = (group + 1) * group_size;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int head = head0 + (lane >> 2) + half * 8, within = column * 8 + (lane & 3) * 2;
            if (head >= end) continue;
            if (partial) {
                float* record = partial + ((static_cast<size_t>(token) * heads + head) * splits + blockIdx.y) * (vdim + 2);
                record[within] = acc[i][2 * half], record[within + 1] = acc[i][2 * half + 1];
                if (within == 0) record[vdim] = tops[head], record[vdim + 1] = sums[head];
            } else {
                const float factor = out_scale / sums[head];
                bf16* target = out + static_cast<size_t>(token) * out_stride + head * vdim + within;
                target[0] = __float2bfloat16_rn(acc[i][2 * half] * factor), target[1] = __float2bfloat16_rn(acc[i][2 * half + 1] * factor);
            }
        }
    }
}

SharedPlan choose_shared_plan(int heads, int kv_heads, int dim, int vdim) {
    if (heads <= 0 || kv_heads <= 0 || dim <= 0 || vdim <= 0 || heads % kv_heads != 0 || static_cast<long long>(kv_heads) * (dim + vdim) > 65536) return SharedPlan{};
    const SharedPlan wide = shared_plan(heads, kv_heads, dim, vdim, 64);
    return wide.keys ? wide : shared_plan(heads, kv_heads, dim, vdim, 32);
}

// Shared memory of the staged kernel, or 0 where it does not serve these sizes.
template <typename T>
int staged_bytes(int dim, int vdim) {
    constexpr int kPer = Word<T>::kElements;
    if (dim % kPer != 0 || vdim % kPer != 0) return 0;
    const long long bytes = (2LL * kTileKeys * (key_stride_words(dim / kPer) + vdim / kPer) + static_cast<long long>(kStagedWarps) * dim) * 4;
    return bytes <= 160 * 1024 ? static_cast<int>(bytes) : 0;
}

template <typename T>
int launch_staged(int bytes, const void* queries, const void* rows, const void* value_pages, void* out, long long out_stride, const int* positions,
                  const int* token_seq, const int* page_rows, int page_stride, int page_tokens, int tokens, int heads, int kv_heads, int dim, int vdim,
                  float scale, int window, int chunk, int sink, float out_scale, const float* distance, int sigmoid_weights, const float* head_offset,
                  const void* gate, long long gate_stride, int gate_per_head, int splits, float* partial, int keep_first, cudaStream_t s) {
    static int allowed = 48 * 1024;
    if (bytes > allowed) {
        cudaError_t status = cudaFuncSetAttribute(masked_attention_staged_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024);
        if (status != cudaSuccess) return static_cast<int>(status);
        allowed = 160 * 1024;
    }
    const int group_size = heads / kv_heads, passes = (group_size + kStagedWarps - 1) / kStagedWarps;
    if ((splits > 1 && !partial) || splits > kMaxSplits) return cudaErrorInvalidValue;
    if (splits <= 1) splits = 1, partial = nullptr;
    tau_launch(masked_attention_staged_kernel<T>, dim3(tokens, kv_heads * passes, splits), dim3(kStagedWarps * 32), bytes, s, static_cast<const T*>(queries),
               static_cast<const T*>(rows), static_cast<const T*>(value_pages), static_cast<T*>(out), out_stride, positions, token_seq, page_rows, page_stride,
               page_tokens, heads, kv_heads, dim, vdim, scale, window, chunk, sink, out_scale, distance, sigmoid_weights, head_offset,
               static_cast<const T*>(gate), gate_stride, gate_per_head, splits, partial, keep_first);
    int status = tau_launch_status();
    if (status != 0 || !partial) return status;
    tau_launch(masked_attention_merge_kernel<T>, dim3(tokens, heads), dim3(128), 0, s, partial, static_cast<T*>(out), out_stride, heads, vdim, splits, out_scale,
               sigmoid_weights, static_cast<const T*>(gate), gate_stride, gate_per_head);
    return tau_launch_status();
}

// out[r, c] = values[r, c] * sigmoid(gate[r, c]); rows of the three any distance apart, `out` may be `values`.
template <typename T>
__global__ void __launch_bounds__(256)
sigmoid_gate_kernel(const T* __restrict__ values, long long values_stride, const T* __restrict__ gate, long long gate_stride, T* __restrict__ out,
                    long long out_stride, int width) {
    grid_dependents_launch();
    grid_dependency_wait();
    const size_t row = blockIdx.x;
    for (int column = threadIdx.x; column < width; column += blockDim.x)
        out[row * out_stride + column] = from_float<T>(to_float(values[row * values_stride + column]) / (1.0f + expf(-to_float(gate[row * gate_stride + column]))));
}

}  // namespace

// 1 where `tau_shared_key_decode` (bfloat16) serves these sizes.
TAU_EXPORT int tau_shared_key_decode_fits(int heads, int kv_heads, int dim, int vdim) { return choose_shared_plan(heads, kv_heads, dim, vdim).keys > 0; }

// Single tokens in bfloat16: queries [tokens, heads, kv_heads * dim] as prepare leaves them with `talk`; the cache in either layout.
TAU_EXPORT int tau_shared_key_decode(const void* queries, const void* rows, const void* value_pages, void* out, long long out_stride, const int* positions,
                                     const int* token_seq, const int* page_rows, int page_stride, int page_tokens, int tokens, int heads, int kv_heads, int dim,
                                     int vdim, float scale, int window, int keep_first, float out_scale, int splits, float* partial, void* stream) {
    if (tokens <= 0) return 0;
    const SharedPlan plan = choose_shared_plan(heads, kv_heads, dim, vdim);
    if (!queries || !rows || !out || !positions || !token_seq || !page_rows || window < 0 || keep_first < 0 || page_tokens <= 0 || plan.keys == 0 ||
        (splits > 1 && !partial) || splits > kMaxSplits)
        return cudaErrorInvalidValue;
    if (splits <= 1) splits = 1, partial = nullptr;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
#define TAU_SHARED(KEYS, ITEMS)                                                                                                                                     \
    {                                                                                                                                                               \
        const cudaError_t status = cudaFuncSetAttribute(shared_key_decode_kernel<KEYS, ITEMS>, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxShared);             \
        if (status != cudaSuccess) return static_cast<int>(status);                                                                                                 \
        tau_launch(shared_key_decode_kernel<KEYS, ITEMS>, dim3(tokens, splits), dim3(kSharedWarps * 32), plan.total, s, static_cast<const bf16*>(queries),           \
                   static_cast<const bf16*>(rows), static_cast<const bf16*>(value_pages), static_cast<bf16*>(out), out_stride, positions, token_seq, page_rows,     \
                   page_stride, page_tokens, heads, kv_heads, dim, vdim, scale, window, keep_first, out_scale, splits, partial);                                     \
    }
    if (plan.keys == 64) {
        if (plan.items <= 8) TAU_SHARED(64, 8)
        else TAU_SHARED(64, 16)
    } else {
        if (plan.items <= 8) TAU_SHARED(32, 8)
        else TAU_SHARED(32, 16)
    }
#undef TAU_SHARED
    const int status = tau_launch_status();
    if (status != 0 || !partial) return status;
    tau_launch(masked_attention_merge_kernel<bf16>, dim3(tokens, heads), dim3(128), 0, s, partial, static_cast<bf16*>(out), out_stride, heads, vdim, splits, out_scale, 0,
               static_cast<const bf16*>(nullptr), 0LL, 0);
    return tau_launch_status();
}

// 1 where `tau_talking_decode` serves these sizes.
TAU_EXPORT int tau_talking_decode_fits(int dtype, int heads, int kv_heads, int dim, int vdim) {
    return dtype == TAU_F32 ? talk_fits<float>(heads, kv_heads, dim, vdim) : dtype == TAU_BF16 ? talk_fits<bf16>(heads, kv_heads, dim, vdim) : 0;
}

// Single tokens: queries [tokens, heads, dim] as prepare leaves them without `talk`; the cache in either layout (see tau_masked_attention).
TAU_EXPORT int tau_talking_decode(int dtype, const void* queries, const void* rows, const void* value_pages, const float* talk, void* out, long long out_stride,
                                  const int* positions, const int* token_seq, const int* page_rows, int page_stride, int page_tokens, int tokens, int heads,
                                  int kv_heads, int dim, int vdim, float scale, int window, int keep_first, float out_scale, int splits, float* partial, void* stream) {
    if (tokens <= 0) return 0;
    if (!queries || !rows || !talk || !out || !positions || !token_seq || !page_rows || window < 0 || keep_first < 0 || page_tokens <= 0) return cudaErrorInvalidValue;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (dtype == TAU_F32)
        return launch_talking_decode<float>(queries, rows, value_pages, talk, out, out_stride, positions, token_seq, page_rows, page_stride, page_tokens, tokens, heads,
                                            kv_heads, dim, vdim, scale, window, keep_first, out_scale, splits, partial, s);
    if (dtype == TAU_BF16)
        return launch_talking_decode<bf16>(queries, rows, value_pages, talk, out, out_stride, positions, token_seq, page_rows, page_stride, page_tokens, tokens, heads,
                                           kv_heads, dim, vdim, scale, window, keep_first, out_scale, splits, partial, s);
    return cudaErrorInvalidValue;
}

TAU_EXPORT int tau_sigmoid_gate(int dtype, const void* values, long long values_stride, const void* gate, long long gate_stride, void* out, long long out_stride,
                                int rows, int width, void* stream) {
    if (rows <= 0) return 0;
    if (!values || !gate || !out || width <= 0) return cudaErrorInvalidValue;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (dtype == TAU_F32)
        tau_launch(sigmoid_gate_kernel<float>, dim3(rows), dim3(256), 0, s, static_cast<const float*>(values), values_stride, static_cast<const float*>(gate), gate_stride,
                   static_cast<float*>(out), out_stride, width);
    else if (dtype == TAU_BF16)
        tau_launch(sigmoid_gate_kernel<bf16>, dim3(rows), dim3(256), 0, s, static_cast<const bf16*>(values), values_stride, static_cast<const bf16*>(gate), gate_stride,
                   static_cast<bf16*>(out), out_stride, width);
    else return cudaErrorInvalidValue;
    return tau_launch_status();
}

TAU_EXPORT int tau_masked_prepare(int dtype, const void* projected, long long projected_stride, const float* q_weight, const float* k_weight, float eps,
                                  const float* frequency, int rotary, float magnitude, void* queries, void* rows, void* value_pages, const int* positions,
                                  const int* token_seq, const int* page_rows, int page_stride, int page_tokens, int tokens, int heads, int kv_heads, int dim, int vdim,
                                  int write_rows, float temperature_coef, int temperature_every, const float* talk, const void* first_values,
                                  long long first_stride, const float* value_share, void* stream) {
    if (tokens <= 0) return 0;
    if (!projected || !queries || !positions || heads <= 0 || kv_heads <= 0 || dim <= 0 || vdim <= 0 || rotary < 0 || rotary > dim || rotary % 2 != 0 ||
        (rotary && !frequency) || (write_rows && (!rows || !token_seq || !page_rows)) || (talk && heads % kv_heads != 0) || (first_values && !value_share))
        return cudaErrorInvalidValue;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    const size_t bytes = static_cast<size_t>((rotary / 2 + 1) / 2 * 2) * sizeof(float2) + (talk ? static_cast<size_t>(heads) * dim * sizeof(float) : 0);
    if (bytes > kMaxShared) return cudaErrorInvalidValue;
#define TAU_PREPARE(T)                                                                                                                            \
    if (bytes > 40 * 1024) {                                                                                                                      \
        const cudaError_t status = cudaFuncSetAttribute(masked_prepare_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxShared);        \
        if (status != cudaSuccess) return static_cast<int>(status);                                                                               \
    }                                                                                                                                             \
    tau_launch(masked_prepare_kernel<T>, dim3(tokens), dim3(kWarps * 32), bytes, s, static_cast<const T*>(projected), projected_stride, q_weight, k_weight, eps, \
               frequency, rotary, magnitude, static_cast<T*>(queries), static_cast<T*>(rows), static_cast<T*>(value_pages), positions, token_seq, page_rows, page_stride, page_tokens, heads,   \
               kv_heads, dim, vdim, write_rows, temperature_coef, temperature_every, talk, static_cast<const T*>(first_values), first_stride, value_share)
    if (dtype == TAU_F32) { TAU_PREPARE(float); }
    else if (dtype == TAU_BF16) { TAU_PREPARE(bf16); }
    else return cudaErrorInvalidValue;
#undef TAU_PREPARE
    return tau_launch_status();
}

// `value_pages` null: `rows` holds one row per position, [pages, page_tokens, kv_heads * (dim + vdim)].  Else keys and values lie in pages
// of their own, `rows` [pages, kv_heads, page_tokens, dim] and `value_pages` [pages, kv_heads, page_tokens, vdim].
TAU_EXPORT int tau_masked_attention(int dtype, const void* queries, const void* rows, const void* value_pages, void* out, long long out_stride, const int* positions,
                                    const int* token_seq, const int* page_rows, int page_stride, int page_tokens, int tokens, int heads, int kv_heads,
                                    int dim, int vdim, float scale, int window, int chunk, int sink, float out_scale, int staged, const float* distance,
                                    int sigmoid_weights, const float* head_offset, const void* gate, long long gate_stride, int gate_per_head, int splits,
                                    float* partial, int keep_first, int shared_keys, void* stream) {
    if (tokens <= 0) return 0;
    if (!queries || !rows || !out || !positions || !token_seq || !page_rows || heads <= 0 || kv_heads <= 0 || heads % kv_heads != 0 || dim <= 0 ||
        vdim <= 0 || vdim > 32 * kMaxOwned || window < 0 || chunk < 0 || (window > 0 && chunk > 0) || (sigmoid_weights && sink) || keep_first < 0)
        return cudaErrorInvalidValue;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    // `staged` (steps of single tokens): the kernel that shares tiles of the cache among a group's heads, where the sizes allow it.
    if (staged && !shared_keys && (dtype == TAU_F32 || dtype == TAU_BF16)) {
        const int staged_size = dtype == TAU_F32 ? staged_bytes<float>(dim, vdim) : staged_bytes<bf16>(dim, vdim);
        if (staged_size > 0) {
            if (dtype == TAU_F32)
                return launch_staged<float>(staged_size, queries, rows, value_pages, out, out_stride, positions, token_seq, page_rows, page_stride, page_tokens,
                                            tokens, heads, kv_heads, dim, vdim, scale, window, chunk, sink, out_scale, distance, sigmoid_weights, head_offset, gate, gate_stride,
                                            gate_per_head, splits, partial, keep_first, s);
            return launch_staged<bf16>(staged_size, queries, rows, value_pages, out, out_stride, positions, token_seq, page_rows, page_stride, page_tokens,
                                       tokens, heads, kv_heads, dim, vdim, scale, window, chunk, sink, out_scale, distance, sigmoid_weights, head_offset, gate, gate_stride,
                                       gate_per_head, splits, partial, keep_first, s);
        }
    }
    const size_t bytes = static_cast<size_t>(kWarps) * dim * (shared_keys ? kv_heads : 1) * sizeof(float);
    if (bytes > kMaxShared) return cudaErrorInvalidValue;
    dim3 grid(tokens, (heads + kWarps - 1) / kWarps);
#define TAU_ATTEND(T)                                                                                                                         \
    if (bytes > 40 * 1024) {                                                                                                                  \
        const cudaError_t status = cudaFuncSetAttribute(masked_attention_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxShared);  \
        if (status != cudaSuccess) return static_cast<int>(status);                                                                           \
    }                                                                                                                                         \
    tau_launch(masked_attention_kernel<T>, grid, dim3(kWarps * 32), bytes, s, static_cast<const T*>(queries), static_cast<const T*>(rows), static_cast<const T*>(value_pages), static_cast<T*>(out), \
               out_stride, positions, token_seq, page_rows, page_stride, page_tokens, heads, kv_heads, dim, vdim, scale, window, chunk, sink, out_scale, distance,         \
               sigmoid_weights, head_offset, static_cast<const T*>(gate), gate_stride, gate_per_head, keep_first, shared_keys)
    if (dtype == TAU_F32) { TAU_ATTEND(float); }
    else if (dtype == TAU_BF16) { TAU_ATTEND(bf16); }
    else return cudaErrorInvalidValue;
#undef TAU_ATTEND
    return tau_launch_status();
}
