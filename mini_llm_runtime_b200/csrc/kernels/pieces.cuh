// A contribution to the residual stream that has not been added up: what routed experts leave (`experts.cu`) for whoever adds it into
// the stream.  Row t is
//     sum_j weights[t, j] * y[row_of_pair[t, j]]      (j = 0 .. top-1 in order; a row of -1 is an identity expert: no row of y)
//   + identity[t] * x[t]                              (with identity experts: the weights of those chosen, times the sub-layer's input)
//   + gate[t] * shared[t]                             (with a shared expert; gate null: as it is)
// in float32.  y null: there is none.
#pragma once

#include "common.cuh"

struct Pieces {
    const float* y;
    long long ldy;
    const int* row_of_pair;
    const float* weights;
    int top;
    const float* shared;
    long long ld_shared;
    const float* gate;
    const void* x;
    long long ld_x;
    int x_bf16;
    const float* identity;
};
constexpr int kMaxPieces = 32;

struct StagedPieces {
    float weight[kMaxPieces];
    long long from[kMaxPieces];       // offset of the piece's row in y, or -1
};

// Leaves a row's weights and places in shared memory; the caller meets at a barrier before `piece_sum`.
__device__ __forceinline__ void stage_pieces(const Pieces& p, int row, StagedPieces& s) {
    if (threadIdx.x < p.top) {
        const int from = __ldcg(p.row_of_pair + static_cast<size_t>(row) * p.top + threadIdx.x);
        s.weight[threadIdx.x] = __ldcg(p.weights + static_cast<size_t>(row) * p.top + threadIdx.x);
        s.from[threadIdx.x] = from < 0 ? -1 : static_cast<long long>(from) * p.ldy;
    }
}

// Columns i .. i + 3 of a row (VEC), or column i alone in `.x`.
template <bool VEC>
__device__ __forceinline__ float4 piece_sum(const Pieces& p, const StagedPieces& s, int row, int i) {
    auto load = [](const float* q, int at) {
        if constexpr (VEC) return __ldcg(reinterpret_cast<const float4*>(q + at));
        else return make_float4(__ldcg(q + at), 0.0f, 0.0f, 0.0f);
    };
    float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    auto add = [&](float w, const float4& e) {
        v.x = fmaf(w, e.x, v.x);
        if constexpr (VEC) { v.y = fmaf(w, e.y, v.y); v.z = fmaf(w, e.z, v.z); v.w = fmaf(w, e.w, v.w); }
    };
#pragma unroll 4
    for (int j = 0; j < p.top; ++j)
        if (s.from[j] >= 0) add(s.weight[j], load(p.y + s.from[j], i));
    if (p.identity) {
        const float w = __ldcg(p.identity + row);
        float e[4] = {};
        const size_t at = static_cast<size_t>(row) * p.ld_x + i;
        if (p.x_bf16) {
            const __nv_bfloat16* x = static_cast<const __nv_bfloat16*>(p.x) + at;
            if constexpr (VEC) mlr_load4(x, e);
            else e[0] = mlr_load(x, 0);
        } else {
            const float* x = static_cast<const float*>(p.x) + at;
            if constexpr (VEC) mlr_load4(x, e);
            else e[0] = mlr_load(x, 0);
        }
        add(w, make_float4(e[0], e[1], e[2], e[3]));
    }
    if (p.shared) add(p.gate ? __ldcg(p.gate + row) : 1.0f, load(p.shared + static_cast<size_t>(row) * p.ld_shared, i));
    return v;
}

static int check_pieces(const Pieces& p, int width, const char* who) {
    MLR_REQUIRE(p.top >= 1 && p.top <= kMaxPieces && p.row_of_pair && p.weights && p.ldy >= width && (!p.shared || p.ld_shared >= width) &&
                    (!p.identity || (p.x && p.ld_x >= width)),
                "%s: a contribution in pieces has 1 to %d pieces a row, with their places, weights and row strides", who, kMaxPieces);
    return 0;
}

// Whether four columns may be read at once.
static bool pieces_aligned(const Pieces& p) {
    const auto fits = [](const void* q, size_t bytes) { return reinterpret_cast<uintptr_t>(q) % bytes == 0; };
    return fits(p.y, 16) && p.ldy % 4 == 0 && (!p.shared || (fits(p.shared, 16) && p.ld_shared % 4 == 0)) &&
           (!p.identity || (fits(p.x, p.x_bf16 ? 8 : 16) && p.ld_x % 4 == 0));
}
