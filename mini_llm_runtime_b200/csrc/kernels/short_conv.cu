// Short causal convolutions over time, per channel, with the last taps - 1 inputs of every request kept as state:
//   y_t = sum_i w[c, i] u_(t - taps + 1 + i) (+ bias), taps [channels, n], the last tap is the current token's, zeros before the start.
//
// `mlr_short_conv` writes silu(y) (what precedes a mixer with a matrix state); `mlr_short_conv_state` moves the state on after a step;
// `mlr_short_conv_step` does both for steps of few rows.
// `mlr_conv_rotate_cache` serves attention: the channels are the projections q | k | v of an attention layer (`MaskedAttentionSpec`); y (no
// activation) of q and k is rotated, q goes to a buffer, k and v to their pages.  With `step` it moves the state on, too.
#include "attention_spec.cuh"
#include "common.cuh"

namespace {

constexpr int kMaxTaps = 16;
constexpr int kConvRows = 8, kConvThreads = 128;

// A thread has V neighbouring channels and walks rows with the last taps - 1 inputs in registers.  N: the number of taps, or 0 for any
// number (then V = 1).  STEP: a block has a segment's rows, all of them, and moves the segment's state on behind them; else it has
// kConvRows rows of the batch, whatever their segments, and the state is read only.
template <typename T, int V, int N, bool STEP>
__global__ void __launch_bounds__(kConvThreads) short_conv_kernel(const T* in, int ld_in, T* out, int ld_out, int channels, int taps,
                                                                  const float* weights, const float* bias, float* state, long long state_stride,
                                                                  const int* segment_info, const int* segment_of_row, int rows) {
    mlr_grid_wait();
    constexpr int kBack = (N ? N : kMaxTaps) - 1;
    const int back = N ? N - 1 : taps - 1;
    const int c = (blockIdx.y * kConvThreads + threadIdx.x) * V;
    if (c >= channels) return;
    float w[kBack + 1][V], past[kBack + 1][V];                  // past[i]: the input that tap i sees
#pragma unroll
    for (int i = 0; i <= kBack; ++i)
#pragma unroll
        for (int j = 0; j < V; ++j) w[i][j] = i <= back ? weights[static_cast<size_t>(c + j) * (back + 1) + i] : 0.0f;
    float shift[V];
#pragma unroll
    for (int j = 0; j < V; ++j) shift[j] = bias ? bias[c + j] : 0.0f;
    int row = STEP ? segment_info[4 * blockIdx.x] : blockIdx.x * kConvRows;
    const int end = STEP ? row + segment_info[4 * blockIdx.x + 1] : min(row + kConvRows, rows);
    int segment = -1;
    float next[V];
    if (row < end) mlr_load_group<V>(in + static_cast<size_t>(row) * ld_in + c, next);
    float* mine = nullptr;
    for (; row < end; ++row) {
        const int now = STEP ? static_cast<int>(blockIdx.x) : segment_of_row[row];
        if (now != segment) {                                   // the inputs before this row: of this step, or from the state
            segment = now;
            const int first = segment_info[4 * segment], j0 = row - first;
            mine = state + static_cast<size_t>(segment_info[4 * segment + 3]) * state_stride + c;
#pragma unroll
            for (int i = 0; i < kBack; ++i)
                if (i < back) {
                    const int m = j0 - back + i;
                    if (m >= 0) mlr_load_group<V>(in + static_cast<size_t>(first + m) * ld_in + c, past[i]);
                    else {
#pragma unroll
                        for (int j = 0; j < V; ++j) past[i][j] = mine[static_cast<size_t>(back + m) * channels + j];
                    }
                }
        }
        float x[V], y[V] = {};
#pragma unroll
        for (int j = 0; j < V; ++j) x[j] = next[j];
        if (row + 1 < end) mlr_load_group<V>(in + static_cast<size_t>(row + 1) * ld_in + c, next);
#pragma unroll
        for (int i = 0; i < kBack; ++i)
            if (i < back) {
#pragma unroll
                for (int j = 0; j < V; ++j) y[j] = fmaf(w[i][j], past[i][j], y[j]);
            }
#pragma unroll
        for (int i = 0; i <= kBack; ++i)
            if (i == back) {
#pragma unroll
                for (int j = 0; j < V; ++j) y[j] = fmaf(w[i][j], x[j], y[j]);
            }
#pragma unroll
        for (int j = 0; j < V; ++j) {
            y[j] += shift[j];
            y[j] = y[j] / (1.0f + expf(-y[j]));
        }
        mlr_store_group<V>(out + static_cast<size_t>(row) * ld_out + c, y);
#pragma unroll
        for (int i = 0; i < kBack; ++i)
            if (i < back) {
#pragma unroll
                for (int j = 0; j < V; ++j) past[i][j] = i + 1 < back ? past[i + 1][j] : x[j];
            }
    }
    if constexpr (STEP) {
        if (mine) {
#pragma unroll
            for (int i = 0; i < kBack; ++i)
                if (i < back) {
#pragma unroll
                    for (int j = 0; j < V; ++j) mine[static_cast<size_t>(i) * channels + j] = past[i][j];
                }
        }
    }
    mlr_grid_dependents_may_start();
}

template <typename T>
__global__ void __launch_bounds__(256) short_conv_state_kernel(const T* in, int ld_in, int channels, int taps, float* state,
                                                               long long state_stride, const int* segment_info) {
    mlr_grid_wait();
    const int segment = blockIdx.x;
    const int first = segment_info[4 * segment], count = segment_info[4 * segment + 1], slot = segment_info[4 * segment + 3];
    float* mine = state + static_cast<size_t>(slot) * state_stride;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < channels; c += gridDim.y * blockDim.x) {
        float kept[kMaxTaps];
        for (int i = 0; i < taps - 1; ++i) kept[i] = mine[static_cast<size_t>(i) * channels + c];
        for (int i = 0; i < taps - 1; ++i) {
            const int m = count - (taps - 1) + i;
            mine[static_cast<size_t>(i) * channels + c] =
                m >= 0 ? mlr_load(in + static_cast<size_t>(first + m) * ld_in, c) : kept[taps - 1 + m];
        }
    }
    mlr_grid_dependents_may_start();
}

// What a thread of the kernel below works on: V pairs of channels (a + j, b + j), j < V, of one head of q, k or v.
struct ConvPairs {
    int kind, head;            // kind 0: q (a map's head), 1: k (kv head * maps + map), 2: v
    int a, b;                  // first values of the pairs within the head
    int channel;               // the head's first channel
    bool rotated, both;        // both: the second values exist (an odd rest has none)
};

template <int V>
__device__ __forceinline__ ConvPairs conv_pairs(const MaskedAttentionSpec& s, int slot) {
    const int half = s.rot_dims / 2, rest = (s.dim - s.rot_dims + 1) / 2, vrest = (s.vdim + 1) / 2;
    const int per_key = half / V + (rest + V - 1) / V, per_value = (vrest + V - 1) / V;
    const int key_heads = s.kv_heads * attention_maps(s);
    ConvPairs p;
    p.rotated = false;
    if (slot < (s.heads + key_heads) * per_key) {
        const int head = slot / per_key, at = slot % per_key;
        p.kind = head < s.heads ? 0 : 1;
        p.head = p.kind == 0 ? head : head - s.heads;
        p.channel = head * s.dim;
        p.rotated = at < half / V;
        if (p.rotated) {
            p.a = at * V;
            p.b = p.a + half;
            p.both = true;
        } else {
            p.a = s.rot_dims + (at - half / V) * V;
            p.b = p.a + rest;
            p.both = p.b < s.dim;
        }
    } else {
        const int left = slot - (s.heads + key_heads) * per_key;
        p.kind = 2;
        p.head = left / per_value;
        p.channel = (s.heads + key_heads) * s.dim + p.head * s.vdim;
        p.a = left % per_value * V;
        p.b = p.a + vrest;
        p.both = p.b < s.vdim;
    }
    return p;
}

template <int V>
__host__ __device__ int conv_slots(const MaskedAttentionSpec& s) {
    const int per_key = s.rot_dims / 2 / V + ((s.dim - s.rot_dims + 1) / 2 + V - 1) / V, per_value = ((s.vdim + 1) / 2 + V - 1) / V;
    return (s.heads + s.kv_heads * attention_maps(s)) * per_key + s.kv_heads * per_value;
}

// A thread walks rows with its channels' last inputs in registers, as in the kernel above (STEP, N: as there).  A row's inputs are loaded
// in the row itself: the form that held the next row's (as above) came out of nvcc 12.9 with the last input in place of the one before it.
template <typename T, int V, int N, bool STEP>
__global__ void __launch_bounds__(kConvThreads) conv_rotate_cache_kernel(const T* in, int ld_in, T* q, int ld_q, int channels, int taps, const float* weights,
                                                                         float* state, long long state_stride, T* cache, int num_pages,
                                                                         const int* positions, const int* segment_info, const int* segment_of_row,
                                                                         const int* block_table, int table_stride, int page_size, int rows,
                                                                         MaskedAttentionSpec s, int* status) {
    mlr_grid_wait();
    constexpr int kBack = (N ? N : kMaxTaps) - 1;
    const int back = N ? N - 1 : taps - 1;
    const int slot = blockIdx.y * kConvThreads + threadIdx.x;
    if (slot >= conv_slots<V>(s)) return;
    const ConvPairs p = conv_pairs<V>(s, slot);
    const int col[2] = {p.channel + p.a, p.channel + (p.both ? p.b : p.a)};
    const int key_row = attention_key_row(s);
    const size_t page_elems = static_cast<size_t>(s.kv_heads) * page_size * (key_row + s.vdim);
    constexpr int E = 2 * V;                                    // a thread's channels: first those from col[0] on, then those from col[1] on
    float w[kBack + 1][E], past[kBack + 1][E], freq[V];         // past[i]: the input that tap i sees
    auto read = [&](float* into, int from) {
        mlr_load_group<V>(in + static_cast<size_t>(from) * ld_in + col[0], into);
        mlr_load_group<V>(in + static_cast<size_t>(from) * ld_in + col[1], into + V);
    };
#pragma unroll
    for (int i = 0; i <= kBack; ++i)
#pragma unroll
        for (int e = 0; e < E; ++e) w[i][e] = i <= back ? weights[static_cast<size_t>(col[e / V] + e % V) * (back + 1) + i] : 0.0f;
#pragma unroll
    for (int j = 0; j < V; ++j) freq[j] = p.rotated ? s.freq[p.a + j] : 0.0f;
    int row = STEP ? segment_info[4 * blockIdx.x] : blockIdx.x * kConvRows;
    const int end = STEP ? row + segment_info[4 * blockIdx.x + 1] : min(row + kConvRows, rows);
    int segment = -1;
    float* mine = nullptr;
    for (; row < end; ++row) {
        const int now = STEP ? static_cast<int>(blockIdx.x) : segment_of_row[row];
        if (now != segment) {                                   // the inputs before this row: of this step, or from the state
            segment = now;
            const int first = segment_info[4 * segment], j0 = row - first;
            mine = state ? state + static_cast<size_t>(segment_info[4 * segment + 3]) * state_stride : nullptr;
#pragma unroll
            for (int i = 0; i < kBack; ++i)
                if (i < back) {
                    const int m = j0 - back + i;
                    if (m >= 0) read(past[i], first + m);
                    else {
#pragma unroll
                        for (int e = 0; e < E; ++e) past[i][e] = mine[static_cast<size_t>(back + m) * channels + col[e / V] + e % V];
                    }
                }
        }
        float x[E], y[E] = {};
        read(x, row);
        const int position = positions[row];
#pragma unroll
        for (int i = 0; i < kBack; ++i)
            if (i < back) {
#pragma unroll
                for (int e = 0; e < E; ++e) y[e] = fmaf(w[i][e], past[i][e], y[e]);
            }
#pragma unroll
        for (int i = 0; i <= kBack; ++i)
            if (i == back) {
#pragma unroll
                for (int e = 0; e < E; ++e) y[e] = fmaf(w[i][e], x[e], y[e]);
            }
#pragma unroll
        for (int i = 0; i < kBack; ++i)
            if (i < back) {
#pragma unroll
                for (int e = 0; e < E; ++e) past[i][e] = i + 1 < back ? past[i + 1][e] : x[e];
            }
        if (p.rotated) {
#pragma unroll
            for (int j = 0; j < V; ++j) {
                float sn, cs;
                sincosf(static_cast<float>(position) * freq[j], &sn, &cs);
                sn *= s.rot_mult;
                cs *= s.rot_mult;
                const float u = y[j], v = y[V + j];
                y[j] = u * cs - v * sn;
                y[V + j] = v * cs + u * sn;
            }
        }
        T* dst = nullptr;
        if (p.kind == 0) {
            dst = q + static_cast<size_t>(row) * ld_q + static_cast<size_t>(p.head) * s.dim;
        } else {
            const int page = block_table[static_cast<size_t>(segment) * table_stride + position / page_size];
            if (page < 0 || page >= num_pages) {
                if (status) atomicOr(status, MLR_STATUS_BAD_PAGE);
            } else {
                T* base = cache + page * page_elems;
                const int maps = key_row / s.dim, in_page = position % page_size;
                if (p.kind == 1) dst = base + (static_cast<size_t>(p.head / maps) * page_size + in_page) * key_row + p.head % maps * s.dim;
                else dst = base + static_cast<size_t>(s.kv_heads) * page_size * key_row + (static_cast<size_t>(p.head) * page_size + in_page) * s.vdim;
            }
        }
        if (dst) {
            mlr_store_group<V>(dst + p.a, y);
            if (p.both) mlr_store_group<V>(dst + p.b, y + V);
        }
    }
    if constexpr (STEP) {
        if (mine) {
#pragma unroll
            for (int i = 0; i < kBack; ++i)
                if (i < back) {
#pragma unroll
                    for (int e = 0; e < E; ++e)
                        if (e < V || p.both) mine[static_cast<size_t>(i) * channels + col[e / V] + e % V] = past[i][e];
                }
        }
    }
    mlr_grid_dependents_may_start();
}

}  // namespace

namespace {
template <bool STEP>
int short_conv(const void* in, int ld_in, void* out, int ld_out, int act_bf16, int channels, int taps, const float* weights, const float* bias,
               float* state, long long state_stride, const int* segment_info, const int* segment_of_row, int blocks, int rows, cudaStream_t stream) {
    const size_t group_bytes = act_bf16 ? 8 : 16;
    const bool wide = taps <= 4 && channels % 4 == 0 && ld_in % 4 == 0 && ld_out % 4 == 0 && reinterpret_cast<uintptr_t>(in) % group_bytes == 0 &&
                      reinterpret_cast<uintptr_t>(out) % group_bytes == 0;
    const dim3 grid(blocks, (channels + kConvThreads * (wide ? 4 : 1) - 1) / (kConvThreads * (wide ? 4 : 1)));
#define MLR_CONV(T, V, N)                                                                                                              \
    mlr_launch((short_conv_kernel<T, V, N, STEP>), dim3(grid), dim3(kConvThreads), 0, stream, static_cast<const T*>(in), ld_in,        \
               static_cast<T*>(out), ld_out, channels, taps, weights, bias, state, state_stride, segment_info, segment_of_row, rows)
#define MLR_CONVS(T)                                                                                                                   \
    do {                                                                                                                               \
        if (!wide) MLR_CONV(T, 1, 0);                                                                                                  \
        else if (taps == 1) MLR_CONV(T, 4, 1);                                                                                         \
        else if (taps == 2) MLR_CONV(T, 4, 2);                                                                                         \
        else if (taps == 3) MLR_CONV(T, 4, 3);                                                                                         \
        else MLR_CONV(T, 4, 4);                                                                                                        \
    } while (0)
    if (act_bf16) MLR_CONVS(__nv_bfloat16);
    else MLR_CONVS(float);
#undef MLR_CONVS
#undef MLR_CONV
    return mlr_launched("short_conv");
}
}  // namespace

// bias: float32 [channels], added before the SiLU, or null.
MLR_API int mlr_short_conv(const void* in, int ld_in, void* out, int ld_out, int act_bf16, int channels, int taps,
                           const float* weights, const float* state, long long state_stride, const int* segment_info,
                           const int* segment_of_row, int rows, const float* bias, cudaStream_t stream) {
    MLR_REQUIRE(channels > 0 && taps >= 1 && taps <= kMaxTaps, "short_conv: %d taps are outside [1, %d]", taps, kMaxTaps);
    MLR_REQUIRE(ld_in >= channels && ld_out >= channels && (taps == 1 || state), "short_conv: bad strides or no state");
    if (rows <= 0) return 0;
    return short_conv<false>(in, ld_in, out, ld_out, act_bf16, channels, taps, weights, bias, const_cast<float*>(state), state_stride, segment_info,
                             segment_of_row, (rows + kConvRows - 1) / kConvRows, rows, stream);
}

// The convolution and the state behind it in one launch: a block walks all rows of a segment (steps of few rows).
MLR_API int mlr_short_conv_step(const void* in, int ld_in, void* out, int ld_out, int act_bf16, int channels, int taps, const float* weights,
                                float* state, long long state_stride, const int* segment_info, int n_segments, const float* bias,
                                cudaStream_t stream) {
    MLR_REQUIRE(channels > 0 && taps >= 1 && taps <= kMaxTaps, "short_conv_step: %d taps are outside [1, %d]", taps, kMaxTaps);
    MLR_REQUIRE(ld_in >= channels && ld_out >= channels && (taps == 1 || state), "short_conv_step: bad strides or no state");
    if (n_segments <= 0) return 0;
    return short_conv<true>(in, ld_in, out, ld_out, act_bf16, channels, taps, weights, bias, state, state_stride, segment_info, nullptr, n_segments, 0,
                            stream);
}

MLR_API int mlr_short_conv_state(const void* in, int ld_in, int act_bf16, int channels, int taps, float* state,
                                 long long state_stride, const int* segment_info, int n_segments, cudaStream_t stream) {
    MLR_REQUIRE(channels > 0 && taps >= 1 && taps <= kMaxTaps, "short_conv_state: %d taps are outside [1, %d]", taps, kMaxTaps);
    if (n_segments <= 0 || taps == 1) return 0;
    const dim3 grid(n_segments, (channels + 255) / 256);
    if (act_bf16)
        mlr_launch((short_conv_state_kernel<__nv_bfloat16>), dim3(grid), dim3(256), 0, stream, static_cast<const __nv_bfloat16*>(in), ld_in,
                   channels, taps, state, state_stride, segment_info);
    else
        mlr_launch((short_conv_state_kernel<float>), dim3(grid), dim3(256), 0, stream, static_cast<const float*>(in), ld_in, channels,
                   taps, state, state_stride, segment_info);
    return mlr_launched("short_conv_state");
}

// in [rows, ld_in]: the projections q [heads * dim] | k [kv_heads * maps * dim] | v [kv_heads * vdim]; weights float32 [channels, taps] of all of
// them; q: the rotated queries [rows, heads * dim]; cache: the layer's pages, keys [kv_head][token][maps * dim] and then values.
// state: float32 [taps - 1, channels] per request slot (unused with one tap).  step: 1 for steps of few rows, whose blocks walk whole segments and
// move the state on; 0: the state is only read (`mlr_short_conv_state` moves it on).
MLR_API int mlr_conv_rotate_cache(const MaskedAttentionSpec* spec, const void* in, int ld_in, void* q, int ld_q, int act_bf16, int taps,
                                  const float* weights, float* state, long long state_stride, void* cache, int num_pages, const int* positions,
                                  const int* segment_info, const int* segment_of_row, const int* block_table, int table_stride, int page_size,
                                  int n_segments, int rows, int step, int* status, cudaStream_t stream) {
    MLR_REQUIRE(spec, "conv_rotate_cache: no description");
    const MaskedAttentionSpec& s = *spec;
    const int channels = s.heads * s.dim + s.kv_heads * (attention_key_row(s) + s.vdim);
    MLR_REQUIRE(s.heads > 0 && s.kv_heads > 0 && s.dim > 0 && s.vdim > 0 && !s.shared_kv && !s.dense_cache, "conv_rotate_cache: bad sizes, or a cache it does not write");
    MLR_REQUIRE(s.rot_dims >= 0 && s.rot_dims % 2 == 0 && s.rot_dims <= s.dim && (s.rot_dims == 0 || s.freq), "conv_rotate_cache: %d rotated values of %d",
                s.rot_dims, s.dim);
    MLR_REQUIRE(taps >= 1 && taps <= kMaxTaps, "conv_rotate_cache: %d taps are outside [1, %d]", taps, kMaxTaps);
    MLR_REQUIRE(in && q && weights && cache && positions && segment_info && segment_of_row && block_table && page_size > 0 && num_pages > 0 &&
                    ld_in >= channels && ld_q >= s.heads * s.dim && (taps == 1 || state), "conv_rotate_cache: bad arguments");
    if (rows <= 0 || n_segments <= 0) return 0;
    const size_t group_bytes = act_bf16 ? 8 : 16;
    const auto fits = [&](const void* p) { return reinterpret_cast<uintptr_t>(p) % group_bytes == 0; };
    const bool wide = taps <= 4 && s.rot_dims % 8 == 0 && s.dim % 8 == 0 && s.vdim % 8 == 0 && ld_in % 4 == 0 && ld_q % 4 == 0 && fits(in) && fits(q) && fits(cache);
    const int slots = wide ? conv_slots<4>(s) : conv_slots<1>(s);
    const dim3 grid(step ? n_segments : (rows + kConvRows - 1) / kConvRows, (slots + kConvThreads - 1) / kConvThreads);
#define MLR_CONV(T, V, N, STEP)                                                                                                        \
    mlr_launch((conv_rotate_cache_kernel<T, V, N, STEP>), dim3(grid), dim3(kConvThreads), 0, stream, static_cast<const T*>(in), ld_in, \
               static_cast<T*>(q), ld_q, channels, taps, weights, taps > 1 ? state : nullptr, state_stride, static_cast<T*>(cache), num_pages, positions, \
               segment_info, segment_of_row, block_table, table_stride, page_size, rows, s, status)
#define MLR_TAPS(T, STEP)                               \
    do {                                                \
        if (!wide) MLR_CONV(T, 1, 0, STEP);             \
        else if (taps == 1) MLR_CONV(T, 4, 1, STEP);    \
        else if (taps == 2) MLR_CONV(T, 4, 2, STEP);    \
        else if (taps == 3) MLR_CONV(T, 4, 3, STEP);    \
        else MLR_CONV(T, 4, 4, STEP);                   \
    } while (0)
    if (act_bf16) {
        if (step) MLR_TAPS(__nv_bfloat16, true);
        else MLR_TAPS(__nv_bfloat16, false);
    } else {
        if (step) MLR_TAPS(float, true);
        else MLR_TAPS(float, false);
    }
#undef MLR_TAPS
#undef MLR_CONV
    return mlr_launched("conv_rotate_cache");
}
