// Mixers that keep a matrix per head and request instead of keys and values: a state S [dim, vdim],
// float32, that every token updates and reads.  One kernel serves the family; what varies between
// designs is a description in host memory (`RecurrenceSpec`):
//
//   activation of q, k and v as they are loaded (in_act): none, or SiLU
//   preparation of q and k (float32, from the projections' output):
//       rotate:  the first rot_dims values turned by position * freq[i] (value i paired with i + rot_dims/2)
//       unit:    x / sqrt(sum(x^2) + unit_eps)
//     then q *= q_mult, k *= k_mult
//   rule, token by token:
//       decay:   S <- decay[head] S + k v^T;                            o = S^T q       (retention)
//       delta:   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;      o = S^T q       (gated delta rule)
//                with g = exp(-exp(a_log[head]) softplus(a + dt_bias[head])), beta = sigmoid(b), from two more
//                columns of the projections' output per head
//       step:    dt = softplus(a + dt_bias[head]);  S <- exp(-exp(a_log[head]) dt) S + dt k v^T;  o = S^T q + skip[head] v
//                (state-space duality), from one more column of the projections' output per head
//     Either of the first two rules may have a decay per head AND key channel instead (channel_decay): it acts on the rows of S, and comes from a
//     product of small rank whose first half is among the projections (decay_rank columns of `side`):
//         z = a W[decay_rank, heads * dim] + bias
//         1: sigmoid(z)^(1 / tau)                            (gated linear attention)
//         2: exp(-exp(a_log[head]) softplus(z))              (channel-wise gated delta rule)
//     and the read-out's gate may be the second half of such a product too (gate_rank columns of `side`).
//   (q, k, v come from one buffer, `proj`; a, b and the gate from another, `side`, which may be the same)
//   read-out:    o / sqrt(mean(o^2) + eps) per head, times a weight [vdim] (optional), times silu(gate)
//                or sigmoid(gate) (optional), times a constant; with norm_all the root mean square is taken over
//                the outputs of all heads of a token together and the weight is [heads * vdim]; with gate_first the gate
//                comes before the norm, which is taken over norm_parts equal parts of all heads' outputs side by side
//
// The columns of S are independent of one another in both rules, so a warp owns a few columns (lanes
// split `dim`), and one block owns one (request, head): it prepares a batch of tokens in shared memory,
// its warps walk the batch token by token, and the block norms and gates the batch's outputs.  The
// state is read at the start and written at the end; a new request's state is zero (the caller zeroes
// the slot).  Everything but the loads of the projections and the store of the result is float32.
#include "common.cuh"

#include <type_traits>

struct RecurrenceSpec {
    const float* freq;         // [rot_dims / 2] or null
    const float* decay;        // [heads] (rule 0)
    const float* a_log;        // [heads] (rule 1)
    const float* dt_bias;      // [heads] (rule 1), or with channel_decay its bias [heads * dim]
    const float* out_weight;   // [vdim] or null
    const float* skip;         // [heads] (rule 2)
    const void* decay_w;       // [decay_rank, heads * dim] in the activations' precision (channel_decay)
    const void* gate_w;        // [gate_rank, heads * vdim] in the activations' precision (gate_rank > 0)
    int heads, qk_heads, dim, vdim;
    int prep;                  // 0 none, 1 rotate, 2 unit
    int rot_dims;
    int rule;                  // 0 decay, 1 delta, 2 step
    int gate_kind;             // 0 none, 1 sigmoid, 2 silu
    int col_q, col_k, col_v;           // first columns of q, k, v in `proj`
    int col_a, col_b, col_gate;        // first columns of the rule's two inputs and of the gate in `side`
    int in_act;                        // 0: q, k, v as projected; 1: through SiLU
    int norm_all;                      // 0: the read-out norms every head alone; 1: all heads of a token together
    int channel_decay;                 // 0: one decay per head; 1: sigmoid(z)^(1 / tau), 2: exp(-exp(a_log) softplus(z)) per key channel
    int decay_rank, gate_rank;         // columns of `side` from col_a on; from col_gate on (0: the gate itself is there)
    int gate_first, norm_parts;        // gate_first: gate, then a norm over each of norm_parts equal parts of [heads * vdim], then the weight [heads * vdim]
    float q_mult, k_mult, unit_eps, eps, out_scale;
    float inv_tau;
};

namespace {

__device__ __forceinline__ float softplus(float x) { return x > 20.0f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float act_in(float x, int kind) { return kind == 1 ? x / (1.0f + expf(-x)) : x; }
// ln(1 + e^x), accurate in both tails.
__device__ __forceinline__ float softplus_exact(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }
// The decay of a key channel from its z.
__device__ __forceinline__ float channel_decay_of(const RecurrenceSpec& s, float z, int head) {
    return s.channel_decay == 1 ? expf(-softplus_exact(-z) * s.inv_tau) : expf(-expf(s.a_log[head]) * softplus_exact(z));
}
// Second half of a product of small rank: sum_r low[r] w[r * stride + c], float32, in the order of r.
template <typename T>
__device__ __forceinline__ float low_rank_dot(const float* low, const T* w, size_t stride, size_t c, int rank) {
    float sum = 0.0f;
    int r = 0;
    for (; r + 8 <= rank; r += 8) {          // eight loads in flight
        float v[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] = mlr_load(w, static_cast<size_t>(r + i) * stride + c);
#pragma unroll
        for (int i = 0; i < 8; ++i) sum = fmaf(low[r + i], v[i], sum);
    }
    for (; r < rank; ++r) sum = fmaf(low[r], mlr_load(w, static_cast<size_t>(r) * stride + c), sum);
    return sum;
}
// The turn of a pair by an angle, with its roundings spelled out: the one-kernel form and the prepare kernel give the same bits.
__device__ __forceinline__ void turn(float u, float v, float cs, float sn, float& a, float& b) {
    a = __fmaf_rn(u, cs, -__fmul_rn(v, sn));
    b = __fmaf_rn(v, cs, __fmul_rn(u, sn));
}

// CH: a decay per key channel (channel_decay).
template <typename T, int R, int COLS, bool CH>
__global__ void __launch_bounds__(1024) linear_recurrence_kernel(const T* proj, int ld, const T* side, int ld_side, T* out, int ld_out, float* state,
                                                                  long long state_stride, const int* segment_info, RecurrenceSpec s,
                                                                  int batch, float* raw) {
    mlr_grid_wait();
    extern __shared__ __align__(16) unsigned char smem[];
    float* qs = reinterpret_cast<float*>(smem);          // [batch][dim]
    float* ks = qs + static_cast<size_t>(batch) * s.dim; // [batch][dim]
    float* vs = ks + static_cast<size_t>(batch) * s.dim; // [batch][vdim]
    float* os = vs + static_cast<size_t>(batch) * s.vdim;  // [batch][vdim]
    float* gs = os + static_cast<size_t>(batch) * s.vdim;  // [batch]
    float* bs = gs + batch;                                 // [batch]
    float* ds = bs + batch;                                 // CH: [batch][dim]
    float* lows = ds + (CH ? static_cast<size_t>(batch) * s.dim : 0);                        // CH: [batch][decay_rank + gate_rank]
    float* gts = lows + (CH ? static_cast<size_t>(batch) * (s.decay_rank + s.gate_rank) : 0);  // CH, gate_rank > 0: [batch][vdim]

    const int segment = blockIdx.x, head = blockIdx.y;
    const int first = segment_info[4 * segment], count = segment_info[4 * segment + 1];
    const int start = segment_info[4 * segment + 2], slot = segment_info[4 * segment + 3];
    const int qk_head = head / (s.heads / s.qk_heads);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    const int threads = blockDim.x;
    const int col0 = warp * COLS;

    float S[COLS][R];
    float* my_state = state + static_cast<size_t>(slot) * state_stride + (static_cast<size_t>(head) * s.vdim) * s.dim;
#pragma unroll
    for (int c = 0; c < COLS; ++c)
#pragma unroll
        for (int r = 0; r < R; ++r) {
            const int d = lane + 32 * r;
            S[c][r] = (col0 + c < s.vdim && d < s.dim) ? my_state[static_cast<size_t>(col0 + c) * s.dim + d] : 0.0f;
        }
    const float decay = !CH && s.rule == 0 ? s.decay[head] : 1.0f;
    const int half = s.rot_dims / 2;

    for (int base = 0; base < count; base += batch) {
        const int n = min(batch, count - base);
        // ---- prepare the batch: q, k, v (and the gates of the rule) as float32
        for (int i = threadIdx.x; i < n * s.dim; i += threads) {
            const int t = i / s.dim, c = i % s.dim;
            const T* row = proj + static_cast<size_t>(first + base + t) * ld;
            qs[i] = act_in(mlr_load(row, s.col_q + qk_head * s.dim + c), s.in_act);
            ks[i] = act_in(mlr_load(row, s.col_k + qk_head * s.dim + c), s.in_act);
        }
        for (int i = threadIdx.x; i < n * s.vdim; i += threads) {
            const int t = i / s.vdim, c = i % s.vdim;
            vs[i] = act_in(mlr_load(proj + static_cast<size_t>(first + base + t) * ld, s.col_v + head * s.vdim + c), s.in_act);
        }
        if (s.rule == 1 && threadIdx.x < n) {
            const T* row = side + static_cast<size_t>(first + base + threadIdx.x) * ld_side;
            const float b = mlr_load(row, s.col_b + head);
            if (!CH) gs[threadIdx.x] = expf(-expf(s.a_log[head]) * softplus(mlr_load(row, s.col_a + head) + s.dt_bias[head]));
            bs[threadIdx.x] = 1.0f / (1.0f + expf(-b));
        }
        if (s.rule == 2 && threadIdx.x < n) {
            const float dt = softplus_exact(mlr_load(side + static_cast<size_t>(first + base + threadIdx.x) * ld_side, s.col_a + head) + s.dt_bias[head]);
            gs[threadIdx.x] = expf(-expf(s.a_log[head]) * dt);
            bs[threadIdx.x] = dt;
        }
        if constexpr (CH) {
            const int ranks = s.decay_rank + s.gate_rank;
            for (int i = threadIdx.x; i < n * ranks; i += threads) {
                const int t = i / ranks, r = i % ranks;
                const T* row = side + static_cast<size_t>(first + base + t) * ld_side;
                lows[i] = mlr_load(row, r < s.decay_rank ? s.col_a + r : s.col_gate + r - s.decay_rank);
            }
        }
        __syncthreads();
        if constexpr (CH) {
            const int ranks = s.decay_rank + s.gate_rank, per_token = s.dim + (s.gate_rank ? s.vdim : 0);
            for (int i = threadIdx.x; i < n * per_token; i += threads) {
                const int t = i / per_token, c = i % per_token;
                const float* low = lows + static_cast<size_t>(t) * ranks;
                if (c < s.dim) {
                    const size_t at = static_cast<size_t>(head) * s.dim + c;
                    const float z = low_rank_dot(low, static_cast<const T*>(s.decay_w), static_cast<size_t>(s.heads) * s.dim, at, s.decay_rank);
                    ds[static_cast<size_t>(t) * s.dim + c] = channel_decay_of(s, z + s.dt_bias[at], head);
                } else {
                    gts[static_cast<size_t>(t) * s.vdim + c - s.dim] =
                        low_rank_dot(low + s.decay_rank, static_cast<const T*>(s.gate_w), static_cast<size_t>(s.heads) * s.vdim,
                                     static_cast<size_t>(head) * s.vdim + c - s.dim, s.gate_rank);
                }
            }
        }
        if (s.prep == 1) {
            for (int i = threadIdx.x; i < n * half; i += threads) {
                const int t = i / half, c = i % half;
                float sn, cs;
                sincosf(static_cast<float>(start + base + t) * s.freq[c], &sn, &cs);
                float* x = qs + static_cast<size_t>(t) * s.dim;
                turn(x[c], x[c + half], cs, sn, x[c], x[c + half]);
                x = ks + static_cast<size_t>(t) * s.dim;
                turn(x[c], x[c + half], cs, sn, x[c], x[c + half]);
            }
            __syncthreads();
            for (int i = threadIdx.x; i < n * s.dim; i += threads) {
                qs[i] = __fmul_rn(qs[i], s.q_mult);
                ks[i] = __fmul_rn(ks[i], s.k_mult);
            }
        } else if (s.prep == 2) {
            for (int vec = warp; vec < 2 * n; vec += warps) {
                float* x = (vec < n ? qs : ks) + static_cast<size_t>(vec < n ? vec : vec - n) * s.dim;
                float sum = 0.0f;
                for (int c = lane; c < s.dim; c += 32) sum = fmaf(x[c], x[c], sum);
                const float inv = 1.0f / sqrtf(mlr_warp_sum(sum) + s.unit_eps);
                const float mult = vec < n ? s.q_mult : s.k_mult;
                for (int c = lane; c < s.dim; c += 32) x[c] = x[c] * inv * mult;
            }
        } else {
            for (int i = threadIdx.x; i < n * s.dim; i += threads) {
                qs[i] *= s.q_mult;
                ks[i] *= s.k_mult;
            }
        }
        __syncthreads();
        // ---- the recurrence: this warp's columns, token by token
        if (col0 < s.vdim) {
            for (int t = 0; t < n; ++t) {
                float kk[R], qq[R], dd[R];
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    const int d = lane + 32 * r;
                    if constexpr (CH) dd[r] = d < s.dim ? ds[static_cast<size_t>(t) * s.dim + d] : 0.0f;
                    kk[r] = d < s.dim ? ks[static_cast<size_t>(t) * s.dim + d] : 0.0f;
                    qq[r] = d < s.dim ? qs[static_cast<size_t>(t) * s.dim + d] : 0.0f;
                }
                float o[COLS];
                if (s.rule != 1) {
                    const float g = !CH && s.rule == 2 ? gs[t] : decay, write = !CH && s.rule == 2 ? bs[t] : 1.0f;
#pragma unroll
                    for (int c = 0; c < COLS; ++c) {
                        const float v = write * (col0 + c < s.vdim ? vs[static_cast<size_t>(t) * s.vdim + col0 + c] : 0.0f);
                        float dot = 0.0f;
#pragma unroll
                        for (int r = 0; r < R; ++r) {
                            S[c][r] = fmaf(CH ? dd[r] : g, S[c][r], kk[r] * v);
                            dot = fmaf(S[c][r], qq[r], dot);
                        }
                        o[c] = dot;
                    }
                } else {
                    const float g = CH ? 1.0f : gs[t], beta = bs[t];
                    float dotk[COLS];
#pragma unroll
                    for (int c = 0; c < COLS; ++c) {
                        float dot = 0.0f;
#pragma unroll
                        for (int r = 0; r < R; ++r) {
                            S[c][r] *= CH ? dd[r] : g;
                            dot = fmaf(S[c][r], kk[r], dot);
                        }
                        dotk[c] = dot;
                    }
#pragma unroll
                    for (int c = 0; c < COLS; ++c) dotk[c] = mlr_warp_sum(dotk[c]);
#pragma unroll
                    for (int c = 0; c < COLS; ++c) {
                        const float v = col0 + c < s.vdim ? vs[static_cast<size_t>(t) * s.vdim + col0 + c] : 0.0f;
                        const float u = beta * (v - dotk[c]);
                        float dot = 0.0f;
#pragma unroll
                        for (int r = 0; r < R; ++r) {
                            S[c][r] = fmaf(kk[r], u, S[c][r]);
                            dot = fmaf(S[c][r], qq[r], dot);
                        }
                        o[c] = dot;
                    }
                }
#pragma unroll
                for (int c = 0; c < COLS; ++c) o[c] = mlr_warp_sum(o[c]);
                if (lane == 0) {
#pragma unroll
                    for (int c = 0; c < COLS; ++c)
                        if (col0 + c < s.vdim) os[static_cast<size_t>(t) * s.vdim + col0 + c] = o[c];
                }
            }
        }
        __syncthreads();
        // ---- read-out of the batch: norm per head, weight, gate; or the plain float32 outputs for a read-out kernel
        for (int t = warp; t < n; t += warps) {
            const float* o = os + static_cast<size_t>(t) * s.vdim;
            if (raw) {
                float* rrow = raw + (static_cast<size_t>(first + base + t) * s.heads + head) * s.vdim;
                if (!CH && s.rule == 2) {
                    for (int c = lane; c < s.vdim; c += 32) rrow[c] = fmaf(s.skip[head], vs[static_cast<size_t>(t) * s.vdim + c], o[c]);
                } else {
                    for (int c = lane; c < s.vdim; c += 32) rrow[c] = o[c];
                }
                continue;
            }
            float inv = 1.0f;
            if (s.eps >= 0.0f) {
                float sum = 0.0f;
                for (int c = lane; c < s.vdim; c += 32) sum = fmaf(o[c], o[c], sum);
                inv = 1.0f / sqrtf(mlr_warp_sum(sum) / static_cast<float>(s.vdim) + s.eps);
            }
            const T* prow = side + static_cast<size_t>(first + base + t) * ld_side;
            T* orow = out + static_cast<size_t>(first + base + t) * ld_out + static_cast<size_t>(head) * s.vdim;
            for (int c = lane; c < s.vdim; c += 32) {
                float value = o[c] * inv;
                if (s.out_weight) value *= s.out_weight[c];
                if (s.gate_kind) {
                    const float g = CH && s.gate_rank ? gts[static_cast<size_t>(t) * s.vdim + c] : mlr_load(prow, s.col_gate + head * s.vdim + c);
                    const float sig = 1.0f / (1.0f + expf(-g));
                    value *= s.gate_kind == 2 ? g * sig : sig;
                }
                mlr_store(orow, c, value * s.out_scale);
            }
        }
        __syncthreads();
    }
    mlr_grid_dependents_may_start();
#pragma unroll
    for (int c = 0; c < COLS; ++c)
#pragma unroll
        for (int r = 0; r < R; ++r) {
            const int d = lane + 32 * r;
            if (col0 + c < s.vdim && d < s.dim) my_state[static_cast<size_t>(col0 + c) * s.dim + d] = S[c][r];
        }
}

// ---- the same in three kernels, for steps of many rows.  The fused kernel above has one block per (request, head):
// a long prompt of one request then runs on a handful of SMs, and every block prepares q and k itself.  Here the
// preparation and the read-out are parallel over rows, and the scan, the only sequential part, has a block per
// (request, head, group of 16 columns of the state).

// q and k of every row, prepared, as float32 [rows, qk_heads * dim] each; for the delta rule also g and beta, for the step rule g and dt [rows, 2 * heads].  zf
// (or null): [rows, heads * dim], z of every key channel without its bias, turned into the channel's decay in place.
constexpr int kPrepareThreads = 256;

template <typename T>
__global__ void __launch_bounds__(kPrepareThreads) recurrence_prepare_kernel(const T* proj, int ld, const T* side, int ld_side, float* qf, float* kf,
                                                                            float* gates, float* zf, const int* positions, RecurrenceSpec s) {
    mlr_grid_wait();
    const int row = blockIdx.x;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    const T* in = proj + static_cast<size_t>(row) * ld;
    const float position = static_cast<float>(positions[row]);
    const int half = s.rot_dims / 2;
    const size_t out_ld = static_cast<size_t>(s.qk_heads) * s.dim;
    for (int vec = warp; vec < 2 * s.qk_heads; vec += warps) {
        const bool is_q = vec < s.qk_heads;
        const int head = is_q ? vec : vec - s.qk_heads;
        const T* x = in + (is_q ? s.col_q : s.col_k) + head * s.dim;
        float* y = (is_q ? qf : kf) + row * out_ld + static_cast<size_t>(head) * s.dim;
        const float mult = is_q ? s.q_mult : s.k_mult;
        if (s.prep == 1) {
            for (int c = lane; c < half; c += 32) {
                float sn, cs;
                sincosf(position * s.freq[c], &sn, &cs);
                const float u = act_in(mlr_load(x, c), s.in_act), v = act_in(mlr_load(x, c + half), s.in_act);
                float a, b;
                turn(u, v, cs, sn, a, b);
                y[c] = __fmul_rn(a, mult);
                y[c + half] = __fmul_rn(b, mult);
            }
            for (int c = s.rot_dims + lane; c < s.dim; c += 32) y[c] = act_in(mlr_load(x, c), s.in_act) * mult;
        } else if (s.prep == 2) {
            float sum = 0.0f;
            for (int c = lane; c < s.dim; c += 32) {
                const float v = act_in(mlr_load(x, c), s.in_act);
                sum = fmaf(v, v, sum);
            }
            const float inv = 1.0f / sqrtf(mlr_warp_sum(sum) + s.unit_eps);
            for (int c = lane; c < s.dim; c += 32) y[c] = act_in(mlr_load(x, c), s.in_act) * inv * mult;
        } else {
            for (int c = lane; c < s.dim; c += 32) y[c] = act_in(mlr_load(x, c), s.in_act) * mult;
        }
    }
    if (s.rule == 1) {
        const T* sd = side + static_cast<size_t>(row) * ld_side;
        for (int h = threadIdx.x; h < s.heads; h += blockDim.x) {
            const float b = mlr_load(sd, s.col_b + h);
            if (!s.channel_decay)
                gates[static_cast<size_t>(row) * 2 * s.heads + h] = expf(-expf(s.a_log[h]) * softplus(mlr_load(sd, s.col_a + h) + s.dt_bias[h]));
            gates[static_cast<size_t>(row) * 2 * s.heads + s.heads + h] = 1.0f / (1.0f + expf(-b));
        }
    }
    if (s.rule == 2) {
        const T* sd = side + static_cast<size_t>(row) * ld_side;
        for (int h = threadIdx.x; h < s.heads; h += blockDim.x) {
            const float dt = softplus_exact(mlr_load(sd, s.col_a + h) + s.dt_bias[h]);
            gates[static_cast<size_t>(row) * 2 * s.heads + h] = expf(-expf(s.a_log[h]) * dt);
            gates[static_cast<size_t>(row) * 2 * s.heads + s.heads + h] = dt;
        }
    }
    if (zf) {
        const int channels = s.heads * s.dim;
        float* z = zf + static_cast<size_t>(row) * channels;
        if (s.dim % 4 == 0) {                    // four channels of one head an access
            for (int c = threadIdx.x * 4; c < channels; c += blockDim.x * 4) {
                const float4 x = __ldcg(reinterpret_cast<const float4*>(z + c)), b = *reinterpret_cast<const float4*>(s.dt_bias + c);
                const int head = c / s.dim;
                *reinterpret_cast<float4*>(z + c) = make_float4(channel_decay_of(s, x.x + b.x, head), channel_decay_of(s, x.y + b.y, head),
                                                                channel_decay_of(s, x.z + b.z, head), channel_decay_of(s, x.w + b.w, head));
            }
        } else {
            for (int c = threadIdx.x; c < channels; c += blockDim.x) z[c] = channel_decay_of(s, __ldcg(z + c) + s.dt_bias[c], c / s.dim);
        }
    }
    mlr_grid_dependents_may_start();
}

// The second halves of the low-rank products of `kChannelRows` rows: df [rows, heads * dim] the decays, gf [rows, heads * vdim] the
// read-out's gate before its sigmoid (gate_rank > 0).  A thread has one channel; the rows' small vectors stand in shared memory.
constexpr int kChannelRows = 16, kChannelThreads = 128;

// V channels a thread (V = 4 where every row of the second matrices starts on a border of four values).
template <typename T, int V>
__global__ void __launch_bounds__(kChannelThreads) recurrence_channel_kernel(const T* side, int ld_side, float* df, float* gf, int rows,
                                                                             RecurrenceSpec s) {
    mlr_grid_wait();
    extern __shared__ __align__(16) float lows[];            // [rank][kChannelRows]
    const int rank_room = s.decay_rank > s.gate_rank ? s.decay_rank : s.gate_rank;
    const int row0 = blockIdx.x * kChannelRows, n = min(kChannelRows, rows - row0);
    constexpr int kPerBlock = kChannelThreads * V;
    const int decays = s.heads * s.dim, decay_blocks = (decays + kPerBlock - 1) / kPerBlock;
    const bool is_gate = static_cast<int>(blockIdx.y) >= decay_blocks;
    const int c = (is_gate ? blockIdx.y - decay_blocks : blockIdx.y) * kPerBlock + threadIdx.x * V;
    const int rank = is_gate ? s.gate_rank : s.decay_rank, col = is_gate ? s.col_gate : s.col_a;
    const int width = is_gate ? s.heads * s.vdim : decays;
    for (int i = threadIdx.x; i < rank * kChannelRows; i += kChannelThreads) {
        const int t = i / rank, r = i % rank;
        lows[r * kChannelRows + t] = t < n ? mlr_load(side + static_cast<size_t>(row0 + t) * ld_side, col + r) : 0.0f;
    }
    __syncthreads();
    if (c < width) {
        const T* w = static_cast<const T*>(is_gate ? s.gate_w : s.decay_w) + c;
        float acc[kChannelRows][V] = {};
        auto add = [&](int r, const float* v) {
#pragma unroll
            for (int t = 0; t < kChannelRows; t += 4) {
                const float4 x4 = *reinterpret_cast<const float4*>(lows + r * kChannelRows + t);
                const float x[4] = {x4.x, x4.y, x4.z, x4.w};
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int j = 0; j < V; ++j) acc[t + i][j] = fmaf(x[i], v[j], acc[t + i][j]);
            }
        };
        constexpr int kAhead = 8 / V;                        // weights in flight
        int r = 0;
        for (; r + kAhead <= rank; r += kAhead) {
            float v[kAhead][V];
#pragma unroll
            for (int i = 0; i < kAhead; ++i) mlr_load_group<V>(w + static_cast<size_t>(r + i) * width, v[i]);
#pragma unroll
            for (int i = 0; i < kAhead; ++i) add(r + i, v[i]);
        }
        for (; r < rank; ++r) {
            float v[V];
            mlr_load_group<V>(w + static_cast<size_t>(r) * width, v);
            add(r, v);
        }
        // The decays' functions are long: they stand once, in a loop over the rows, whose sums wait in shared memory.
        float* zs = lows + rank_room * kChannelRows + threadIdx.x * V;        // [kChannelRows][threads * V], a thread's own columns
#pragma unroll
        for (int t = 0; t < kChannelRows; ++t) mlr_store_group<V>(zs + t * kPerBlock, acc[t]);
        float* out = (is_gate ? gf : df) + static_cast<size_t>(row0) * width + c;
        float bias[V] = {};
        if (!is_gate) {
#pragma unroll
            for (int j = 0; j < V; ++j) bias[j] = s.dt_bias[c + j];
        }
#pragma unroll 1
        for (int t = 0; t < n; ++t) {
            float z[V];
#pragma unroll
            for (int j = 0; j < V; ++j) z[j] = zs[t * kPerBlock + j];
            if (!is_gate) {
#pragma unroll
                for (int j = 0; j < V; ++j) z[j] = channel_decay_of(s, z[j] + bias[j], (c + j) / s.dim);
            }
            mlr_store_group<V>(out + static_cast<size_t>(t) * width, z);
        }
    }
    mlr_grid_dependents_may_start();
}

constexpr int kScanWarps = 4, kScanCols = 4, kScanBlockCols = kScanWarps * kScanCols;

template <typename T, int R, bool CH>
__global__ void __launch_bounds__(kScanWarps * 32) recurrence_scan_kernel(const float* qf, const float* kf, const float* df, const float* gates, const T* proj,
                                                                          int ld, float* obuf, float* state, long long state_stride,
                                                                          const int* segment_info, RecurrenceSpec s, int batch) {
    mlr_grid_wait();
    extern __shared__ __align__(16) unsigned char smem[];
    const size_t stage = static_cast<size_t>(batch) * s.dim;
    float* qs = reinterpret_cast<float*>(smem);                // [2][batch][dim]: a batch is copied while the one before is walked
    float* ks = qs + 2 * stage;                                // [2][batch][dim]
    float* vs = ks + 2 * stage;                                // [batch][16]
    float* os = vs + static_cast<size_t>(batch) * kScanBlockCols;   // [batch][16]
    float* gs = os + static_cast<size_t>(batch) * kScanBlockCols;   // [batch]
    float* bs = gs + batch;                                    // [batch]
    float* ds = gs + ((2 * batch + 3) & ~3);                   // CH: [2][batch][dim], decays per channel
    const size_t d_ld = static_cast<size_t>(s.heads) * s.dim;
    const int segment = blockIdx.x, head = blockIdx.y, block_col = blockIdx.z * kScanBlockCols;
    const int first = segment_info[4 * segment], count = segment_info[4 * segment + 1], slot = segment_info[4 * segment + 3];
    const int qk_head = head / (s.heads / s.qk_heads);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int col0 = block_col + warp * kScanCols;
    const size_t qk_ld = static_cast<size_t>(s.qk_heads) * s.dim;
    const size_t o_ld = static_cast<size_t>(s.heads) * s.vdim;
    const bool wide = s.dim % 4 == 0;                          // rows of q and k start on 16-byte borders

    float S[kScanCols][R];
    float* my_state = state + static_cast<size_t>(slot) * state_stride + (static_cast<size_t>(head) * s.vdim) * s.dim;
#pragma unroll
    for (int c = 0; c < kScanCols; ++c)
#pragma unroll
        for (int r = 0; r < R; ++r) {
            const int d = lane + 32 * r;
            S[c][r] = (col0 + c < s.vdim && d < s.dim) ? my_state[static_cast<size_t>(col0 + c) * s.dim + d] : 0.0f;
        }
    const float decay = !CH && s.rule == 0 ? s.decay[head] : 1.0f;

    constexpr int kVPerThread = 32 * kScanBlockCols / (kScanWarps * 32);     // batch <= 32
    float v_next[kVPerThread], g_next = 0.0f, b_next = 0.0f;
    // Starts the copies of a batch's q and k into a stage and loads its v, g and beta into registers.
    auto fetch = [&](int base, int into) {
        const int n = min(batch, count - base);
        const float* qsrc = qf + static_cast<size_t>(first + base) * qk_ld + static_cast<size_t>(qk_head) * s.dim;
        const float* ksrc = kf + static_cast<size_t>(first + base) * qk_ld + static_cast<size_t>(qk_head) * s.dim;
        float* qdst = qs + into * stage;
        float* kdst = ks + into * stage;
        const float* dsrc = CH ? df + static_cast<size_t>(first + base) * d_ld + static_cast<size_t>(head) * s.dim : nullptr;
        float* ddst = ds + into * stage;
        if (wide) {
            const int per_row = s.dim / 4;
            for (int i = threadIdx.x; i < n * per_row; i += blockDim.x) {
                const int t = i / per_row, c = (i % per_row) * 4;
                mlr_async_copy16(qdst + static_cast<size_t>(t) * s.dim + c, qsrc + t * qk_ld + c);
                mlr_async_copy16(kdst + static_cast<size_t>(t) * s.dim + c, ksrc + t * qk_ld + c);
                if constexpr (CH) mlr_async_copy16(ddst + static_cast<size_t>(t) * s.dim + c, dsrc + t * d_ld + c);
            }
        } else {
            for (int i = threadIdx.x; i < n * s.dim; i += blockDim.x) {
                const int t = i / s.dim, c = i % s.dim;
                mlr_async_copy4(qdst + static_cast<size_t>(t) * s.dim + c, qsrc + t * qk_ld + c);
                mlr_async_copy4(kdst + static_cast<size_t>(t) * s.dim + c, ksrc + t * qk_ld + c);
                if constexpr (CH) mlr_async_copy4(ddst + static_cast<size_t>(t) * s.dim + c, dsrc + t * d_ld + c);
            }
        }
        mlr_async_commit();
#pragma unroll
        for (int j = 0; j < kVPerThread; ++j) {
            const int i = threadIdx.x + j * kScanWarps * 32;
            const int t = i / kScanBlockCols, c = block_col + i % kScanBlockCols;
            v_next[j] = (t < n && c < s.vdim) ? mlr_load(proj + static_cast<size_t>(first + base + t) * ld, s.col_v + head * s.vdim + c) : 0.0f;
        }
        if (s.rule != 0 && threadIdx.x < n) {
            if constexpr (!CH) g_next = __ldcg(gates + static_cast<size_t>(first + base + threadIdx.x) * 2 * s.heads + head);
            b_next = __ldcg(gates + static_cast<size_t>(first + base + threadIdx.x) * 2 * s.heads + s.heads + head);
        }
    };

    fetch(0, 0);
    int current = 0;
    for (int base = 0; base < count; base += batch, current ^= 1) {
        const int n = min(batch, count - base);
        __syncthreads();                    // the batch before has been walked and written out
#pragma unroll
        for (int j = 0; j < kVPerThread; ++j) {
            const int i = threadIdx.x + j * kScanWarps * 32;
            if (i < batch * kScanBlockCols) vs[i] = act_in(v_next[j], s.in_act);
        }
        if (threadIdx.x < batch) {
            gs[threadIdx.x] = g_next;
            bs[threadIdx.x] = b_next;
        }
        mlr_async_wait();
        __syncthreads();
        if (base + batch < count) fetch(base + batch, current ^ 1);
        const float* qnow = qs + current * stage;
        const float* know = ks + current * stage;
        const float* dnow = ds + current * stage;
        for (int t = 0; t < n; ++t) {
            float kk[R], qq[R], dd[R];
#pragma unroll
            for (int r = 0; r < R; ++r) {
                const int d = lane + 32 * r;
                if constexpr (CH) dd[r] = d < s.dim ? dnow[static_cast<size_t>(t) * s.dim + d] : 0.0f;
                kk[r] = d < s.dim ? know[static_cast<size_t>(t) * s.dim + d] : 0.0f;
                qq[r] = d < s.dim ? qnow[static_cast<size_t>(t) * s.dim + d] : 0.0f;
            }
            float o[kScanCols];
            if (s.rule != 1) {
                const float g = !CH && s.rule == 2 ? gs[t] : decay, write = !CH && s.rule == 2 ? bs[t] : 1.0f;
#pragma unroll
                for (int c = 0; c < kScanCols; ++c) {
                    const float v = write * vs[t * kScanBlockCols + warp * kScanCols + c];
                    float dot = 0.0f;
#pragma unroll
                    for (int r = 0; r < R; ++r) {
                        S[c][r] = fmaf(CH ? dd[r] : g, S[c][r], kk[r] * v);
                        dot = fmaf(S[c][r], qq[r], dot);
                    }
                    o[c] = dot;
                }
            } else {
                const float g = CH ? 1.0f : gs[t], beta = bs[t];
                float dotk[kScanCols];
#pragma unroll
                for (int c = 0; c < kScanCols; ++c) {
                    float dot = 0.0f;
#pragma unroll
                    for (int r = 0; r < R; ++r) {
                        S[c][r] *= CH ? dd[r] : g;
                        dot = fmaf(S[c][r], kk[r], dot);
                    }
                    dotk[c] = dot;
                }
#pragma unroll
                for (int c = 0; c < kScanCols; ++c) dotk[c] = mlr_warp_sum(dotk[c]);
#pragma unroll
                for (int c = 0; c < kScanCols; ++c) {
                    const float v = vs[t * kScanBlockCols + warp * kScanCols + c];
                    const float u = beta * (v - dotk[c]);
                    float dot = 0.0f;
#pragma unroll
                    for (int r = 0; r < R; ++r) {
                        S[c][r] = fmaf(kk[r], u, S[c][r]);
                        dot = fmaf(S[c][r], qq[r], dot);
                    }
                    o[c] = dot;
                }
            }
#pragma unroll
            for (int c = 0; c < kScanCols; ++c) o[c] = mlr_warp_sum(o[c]);
            if (lane == 0) {
#pragma unroll
                for (int c = 0; c < kScanCols; ++c) os[t * kScanBlockCols + warp * kScanCols + c] = o[c];
            }
        }
        __syncthreads();
        for (int i = threadIdx.x; i < n * kScanBlockCols; i += blockDim.x) {
            const int t = i / kScanBlockCols, c = block_col + i % kScanBlockCols;
            const float o = !CH && s.rule == 2 ? fmaf(s.skip[head], vs[i], os[i]) : os[i];
            if (c < s.vdim) obuf[static_cast<size_t>(first + base + t) * o_ld + static_cast<size_t>(head) * s.vdim + c] = o;
        }
    }
    mlr_grid_dependents_may_start();     // only now: blocks of the next grid that wait on this SM slow the walk
#pragma unroll
    for (int c = 0; c < kScanCols; ++c)
#pragma unroll
        for (int r = 0; r < R; ++r) {
            const int d = lane + 32 * r;
            if (col0 + c < s.vdim && d < s.dim) my_state[static_cast<size_t>(col0 + c) * s.dim + d] = S[c][r];
        }
}

// The same walk for head sizes DIM that are a multiple of 32, with sixteen lanes a column: a lane keeps DIM / 16 state values of ONE column,
// eight warps share the block's 16 columns (two warps a scheduler hide one another's waits).  Four tokens at a time: the sums of their
// outputs over a column's lanes are exchanged together (five exchanges for four tokens), and nothing is stored to shared memory in
// between; a token's k, q and decays are loaded from shared memory while the token before it is walked.
constexpr int kColumnLanes = 16, kColumnWarps = kScanBlockCols * kColumnLanes / 32;

// NC: columns of the state a lane works on (column c and c + 16): two halve the reading of k and q where blocks outnumber the SMs.
template <typename T, int DIM, int RULE, bool CH, int NC>
__global__ void __launch_bounds__(kColumnWarps * 32) recurrence_scan16_kernel(const float* qf, const float* kf, const float* df, const float* gates,
                                                                            const T* proj, int ld, float* obuf, float* state, long long state_stride,
                                                                            const int* segment_info, RecurrenceSpec s, int batch) {
    mlr_grid_wait();
    constexpr int kThreads = kColumnWarps * 32, E = DIM / kColumnLanes, V = E % 4 == 0 ? 4 : 2;       // V: values an access
    constexpr int kCols = kScanBlockCols * NC;
    extern __shared__ __align__(16) unsigned char smem[];
    const int stage = batch * DIM;                             // batch: a multiple of 4, at most 32
    float* qs = reinterpret_cast<float*>(smem);                // [2][batch][DIM]: a batch is copied while the one before is walked
    float* ks = qs + 2 * stage;                                // [2][batch][DIM]
    float* ds = ks + 2 * stage;                                // CH: [2][batch][DIM], decays per channel
    float* vs = ds + (CH ? 2 * stage : 0);                     // [kCols][batch]
    float* os = vs + batch * kCols;                   // [batch][kCols]
    float* gs = os + batch * kCols;                   // [batch]
    float* bs = gs + batch;                                    // [batch]
    const int segment = blockIdx.x, head = blockIdx.y, block_col = blockIdx.z * kCols;
    const int first = segment_info[4 * segment], count = segment_info[4 * segment + 1], slot = segment_info[4 * segment + 3];
    const int qk_head = head / (s.heads / s.qk_heads);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int sub = lane & (kColumnLanes - 1), my_col = warp * (32 / kColumnLanes) + lane / kColumnLanes;
    const size_t qk_ld = static_cast<size_t>(s.qk_heads) * DIM, d_ld = static_cast<size_t>(s.heads) * DIM;
    const size_t o_ld = static_cast<size_t>(s.heads) * s.vdim;
    const float decay = !CH && RULE == 0 ? s.decay[head] : 1.0f;

    float S[NC][E];
    float* my_state = state + static_cast<size_t>(slot) * state_stride + (static_cast<size_t>(head) * s.vdim + block_col + my_col) * DIM;
    auto live = [&](int n) { return block_col + my_col + n * kScanBlockCols < s.vdim; };
    // Value j of a lane is value V * (16 * (j / V) + sub) + j % V of the head: sixteen lanes read consecutive bytes.
    auto place = [&](int j) { return V * (kColumnLanes * (j / V) + sub) + j % V; };
#pragma unroll
    for (int n = 0; n < NC; ++n)
#pragma unroll
        for (int j = 0; j < E; ++j) S[n][j] = live(n) ? my_state[n * kScanBlockCols * DIM + place(j)] : 0.0f;

    constexpr int kVPerThread = 32 * kCols / kThreads;
    T v_next[kVPerThread];                // as loaded: a conversion right behind the load would wait for it
    float g_next = 0.0f, b_next = 0.0f;
    // Starts the copies of a batch's q, k and decays into a stage and loads its v, g and beta into registers.
    auto fetch = [&](int base, int into) {
        const int n = min(batch, count - base);
        const float* qsrc = qf + static_cast<size_t>(first + base) * qk_ld + static_cast<size_t>(qk_head) * DIM;
        const float* ksrc = kf + static_cast<size_t>(first + base) * qk_ld + static_cast<size_t>(qk_head) * DIM;
        const float* dsrc = CH ? df + static_cast<size_t>(first + base) * d_ld + static_cast<size_t>(head) * DIM : nullptr;
        float* qdst = qs + into * stage;
        float* kdst = ks + into * stage;
        float* ddst = ds + into * stage;
        constexpr int kPerRow = DIM / 4;
        for (int i = threadIdx.x; i < n * kPerRow; i += kThreads) {
            const int t = i / kPerRow, c = (i % kPerRow) * 4;
            mlr_async_copy16(qdst + t * DIM + c, qsrc + t * qk_ld + c);
            mlr_async_copy16(kdst + t * DIM + c, ksrc + t * qk_ld + c);
            if constexpr (CH) mlr_async_copy16(ddst + t * DIM + c, dsrc + t * d_ld + c);
        }
        mlr_async_commit();
#pragma unroll
        for (int j = 0; j < kVPerThread; ++j) {
            const int i = threadIdx.x + j * kThreads;
            const int t = i / kCols, c = block_col + i % kCols;
            v_next[j] = proj[(t < n && c < s.vdim) ? static_cast<size_t>(first + base + t) * ld + s.col_v + head * s.vdim + c : 0];
        }
        if (RULE != 0 && threadIdx.x < n) {
            const float* g = gates + static_cast<size_t>(first + base + threadIdx.x) * 2 * s.heads + head;
            if constexpr (!CH) g_next = __ldcg(g);
            b_next = __ldcg(g + s.heads);
        }
    };

    struct Token {
        float k[E], q[E], d[CH ? E : 1];
    };
    fetch(0, 0);
    int current = 0;
    for (int base = 0; base < count; base += batch, current ^= 1) {
        const int n = min(batch, count - base);
        __syncthreads();                    // the batch before has been walked and written out
#pragma unroll
        for (int j = 0; j < kVPerThread; ++j) {
            const int i = threadIdx.x + j * kThreads;
            if (i < batch * kCols) vs[i % kCols * batch + i / kCols] = act_in(mlr_load(&v_next[j], 0), s.in_act);
        }
        if (RULE != 0 && threadIdx.x < batch) {
            gs[threadIdx.x] = g_next;
            bs[threadIdx.x] = b_next;
        }
        mlr_async_wait();
        __syncthreads();
        if (base + batch < count) fetch(base + batch, current ^ 1);
        const float* qnow = qs + current * stage + V * sub;
        const float* know = ks + current * stage + V * sub;
        const float* dnow = ds + current * stage + V * sub;
        auto load = [&](Token& x, int t) {
            auto vector = [&](float* into, const float* from) {
#pragma unroll
                for (int e = 0; e < E / V; ++e) {
                    if constexpr (V == 4) {
                        const float4 y = *reinterpret_cast<const float4*>(from + t * DIM + V * kColumnLanes * e);
                        into[4 * e] = y.x; into[4 * e + 1] = y.y; into[4 * e + 2] = y.z; into[4 * e + 3] = y.w;
                    } else {
                        const float2 y = *reinterpret_cast<const float2*>(from + t * DIM + V * kColumnLanes * e);
                        into[2 * e] = y.x; into[2 * e + 1] = y.y;
                    }
                }
            };
            vector(x.k, know);
            if constexpr (CH) vector(x.d, dnow);
            vector(x.q, qnow);
        };
        Token tokens[2];
        load(tokens[0], 0);
        // GUARDED: the batch's last, incomplete group of four.  Rows past the batch are not read: a token's successor is at most the last.
        auto walk4 = [&](int t0, auto guarded) {
            constexpr bool kGuarded = decltype(guarded)::value;
            float v[NC][4];
#pragma unroll
            for (int m = 0; m < NC; ++m) {
                const float4 v4 = *reinterpret_cast<const float4*>(vs + (my_col + m * kScanBlockCols) * batch + t0);
                v[m][0] = v4.x; v[m][1] = v4.y; v[m][2] = v4.z; v[m][3] = v4.w;
            }
            [[maybe_unused]] float g[4] = {decay, decay, decay, decay}, beta[4] = {};
            if constexpr (RULE != 0) {
                const float4 b4 = *reinterpret_cast<const float4*>(bs + t0);
                beta[0] = b4.x; beta[1] = b4.y; beta[2] = b4.z; beta[3] = b4.w;
                if constexpr (!CH) {
                    const float4 g4 = *reinterpret_cast<const float4*>(gs + t0);
                    g[0] = g4.x; g[1] = g4.y; g[2] = g4.z; g[3] = g4.w;
                }
            }
            float dots[NC][4];
#pragma unroll
            for (int u = 0; u < 4; ++u) {
#pragma unroll
                for (int m = 0; m < NC; ++m) dots[m][u] = 0.0f;
                if (!kGuarded || t0 + u < n) {
                    const Token& x = tokens[u & 1];
                    load(tokens[(u + 1) & 1], u < 3 && !kGuarded ? t0 + u + 1 : min(t0 + u + 1, n - 1));
#pragma unroll
                    for (int m = 0; m < NC; ++m) {
                        float write = RULE == 2 ? beta[u] * v[m][u] : v[m][u];
                        if constexpr (RULE != 1) {
#pragma unroll
                            for (int j = 0; j < E; ++j) S[m][j] = fmaf(CH ? x.d[CH ? j : 0] : g[u], S[m][j], x.k[j] * write);
                        } else {
                            float c[2] = {};
#pragma unroll
                            for (int j = 0; j < E; ++j) {
                                S[m][j] *= CH ? x.d[CH ? j : 0] : g[u];
                                c[j & 1] = fmaf(S[m][j], x.k[j], c[j & 1]);
                            }
                            float held = c[0] + c[1];
#pragma unroll
                            for (int step = 1; step < kColumnLanes; step *= 2) held += __shfl_xor_sync(0xffffffffu, held, step);
                            write = beta[u] * (write - held);
#pragma unroll
                            for (int j = 0; j < E; ++j) S[m][j] = fmaf(x.k[j], write, S[m][j]);
                        }
                        float o[2] = {};
#pragma unroll
                        for (int j = 0; j < E; ++j) o[j & 1] = fmaf(S[m][j], x.q[j], o[j & 1]);
                        dots[m][u] = o[0] + o[1];
                    }
                }
            }
            // Lanes with sub % 4 == u end up with the sum of token t0 + u.
            const bool odd = sub & 1, high = sub & 2;
#pragma unroll
            for (int m = 0; m < NC; ++m) {
                const float even_pair = (odd ? dots[m][1] : dots[m][0]) + __shfl_xor_sync(0xffffffffu, odd ? dots[m][0] : dots[m][1], 1);
                const float odd_pair = (odd ? dots[m][3] : dots[m][2]) + __shfl_xor_sync(0xffffffffu, odd ? dots[m][2] : dots[m][3], 1);
                float sum = (high ? odd_pair : even_pair) + __shfl_xor_sync(0xffffffffu, high ? even_pair : odd_pair, 2);
                sum += __shfl_xor_sync(0xffffffffu, sum, 4);
                sum += __shfl_xor_sync(0xffffffffu, sum, 8);
                if (sub < 4 && (!kGuarded || t0 + sub < n)) os[(t0 + sub) * kCols + my_col + m * kScanBlockCols] = sum;
            }
        };
        for (int t0 = 0; t0 < n; t0 += 4) {
            if (t0 + 4 <= n) walk4(t0, std::false_type{});      // whole groups carry no per-token conditions
            else walk4(t0, std::true_type{});
        }
        __syncthreads();
        for (int i = threadIdx.x; i < n * kCols; i += kThreads) {
            const int t = i / kCols, c = block_col + i % kCols;
            const float o = RULE == 2 ? fmaf(s.skip[head], vs[i % kCols * batch + t], os[i]) : os[i];
            if (c < s.vdim) obuf[static_cast<size_t>(first + base + t) * o_ld + static_cast<size_t>(head) * s.vdim + c] = o;
        }
    }
    mlr_grid_dependents_may_start();     // only now: blocks of the next grid that wait on this SM slow the walk
#pragma unroll
    for (int n = 0; n < NC; ++n)
        if (live(n)) {
#pragma unroll
            for (int j = 0; j < E; ++j) my_state[n * kScanBlockCols * DIM + place(j)] = S[n][j];
        }
}


// Norm per head, weight, gate and the constant on the scan's float32 outputs [rows, heads * vdim].  gf: the gate's values in
// float32 [rows, heads * vdim] when they come of a low-rank product, else null and the gate is in `side`.
// VEC: four values an access, a head's values held in registers between the sum and the result (vdim a multiple of 4, at most 256).
constexpr int kReadoutThreads = 256;

template <typename T, bool VEC>
__global__ void __launch_bounds__(kReadoutThreads) recurrence_readout_kernel(const float* obuf, const T* side, int ld_side, const float* gf, T* out,
                                                                            int ld_out, RecurrenceSpec s) {
    mlr_grid_wait();
    constexpr int V = VEC ? 4 : 1, kHeld = 256 / (32 * V);
    const int row = blockIdx.x;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    __shared__ float scratch[32];
    float inv_all = 1.0f;
    if (s.norm_all && s.eps >= 0.0f) {
        const int total = s.heads * s.vdim;
        const float* o = obuf + static_cast<size_t>(row) * total;
        float sum = 0.0f;
        for (int c = threadIdx.x; c < total; c += blockDim.x) {
            const float v = __ldcg(o + c);
            sum = fmaf(v, v, sum);
        }
        inv_all = 1.0f / sqrtf(mlr_block_sum(sum, scratch) / static_cast<float>(total) + s.eps);
    }
    for (int head = warp; head < s.heads; head += warps) {
        const float* o = obuf + (static_cast<size_t>(row) * s.heads + head) * s.vdim;
        float held[kHeld][V];
#pragma unroll
        for (int i = 0; i < kHeld; ++i) {
            const int c = (i * 32 + lane) * V;
            if (c < s.vdim) mlr_load_group<V>(o + c, held[i]);
        }
        float inv = inv_all;
        if (s.eps >= 0.0f && !s.norm_all) {
            float sum = 0.0f;
#pragma unroll
            for (int i = 0; i < kHeld; ++i)
                if ((i * 32 + lane) * V < s.vdim) {
#pragma unroll
                    for (int j = 0; j < V; ++j) sum = fmaf(held[i][j], held[i][j], sum);
                }
            inv = 1.0f / sqrtf(mlr_warp_sum(sum) / static_cast<float>(s.vdim) + s.eps);
        }
        const T* grow = side + static_cast<size_t>(row) * ld_side + s.col_gate + head * s.vdim;
        const float* gfrow = gf + (static_cast<size_t>(row) * s.heads + head) * s.vdim;
        T* orow = out + static_cast<size_t>(row) * ld_out + static_cast<size_t>(head) * s.vdim;
#pragma unroll
        for (int i = 0; i < kHeld; ++i) {
            const int c = (i * 32 + lane) * V;
            if (c >= s.vdim) break;
            float g[V] = {};
            if (s.gate_kind) {
                if (gf) mlr_load_group<V>(gfrow + c, g);
                else mlr_load_group<V>(grow + c, g);
            }
            float value[V];
#pragma unroll
            for (int j = 0; j < V; ++j) {
                value[j] = held[i][j] * inv;
                if (s.out_weight) value[j] *= s.out_weight[s.norm_all ? head * s.vdim + c + j : c + j];
                if (s.gate_kind) {
                    const float sig = 1.0f / (1.0f + expf(-g[j]));
                    value[j] *= s.gate_kind == 2 ? g[j] * sig : sig;
                }
                value[j] *= s.out_scale;
            }
            mlr_store_group<V>(orow + c, value);
        }
    }
    mlr_grid_dependents_may_start();
}

// The read-out with the gate in front: o times its gate (`side`), each of s.norm_parts equal parts of a token's outputs (all heads side
// by side) over its own root mean square, times the weight [heads * vdim] and the constant.  A block per row, the gated values in
// shared memory: [heads * vdim] and one sum per part.
template <typename T, int V>
__global__ void __launch_bounds__(kReadoutThreads) recurrence_parts_readout_kernel(const float* obuf, const T* side, int ld_side, T* out, int ld_out,
                                                                                  RecurrenceSpec s) {
    mlr_grid_wait();
    extern __shared__ __align__(16) float gated[];
    __shared__ float scratch[32];
    const int row = blockIdx.x, total = s.heads * s.vdim, part = total / s.norm_parts;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    float* inv = gated + (total + 3) / 4 * 4;
    const float* o = obuf + static_cast<size_t>(row) * total;
    const T* grow = side + static_cast<size_t>(row) * ld_side + s.col_gate;
    float mine = 0.0f;
    for (int c = threadIdx.x * V; c < total; c += blockDim.x * V) {
        float v[V], g[V];
        mlr_load_group<V>(o + c, v);
        if (s.gate_kind) {
            mlr_load_group<V>(grow + c, g);
#pragma unroll
            for (int j = 0; j < V; ++j) {
                const float sig = 1.0f / (1.0f + expf(-g[j]));
                v[j] *= s.gate_kind == 2 ? g[j] * sig : sig;
            }
        }
#pragma unroll
        for (int j = 0; j < V; ++j) mine = fmaf(v[j], v[j], mine);
        mlr_store_group<V>(gated + c, v);
    }
    if (s.norm_parts == 1) {
        const float sum = mlr_block_sum(mine, scratch);
        if (threadIdx.x == 0) inv[0] = 1.0f / sqrtf(sum / static_cast<float>(part) + s.eps);
        __syncthreads();
    } else {
        __syncthreads();
        for (int g = warp; g < s.norm_parts; g += warps) {
            float sum = 0.0f;
            for (int c = lane; c < part; c += 32) sum = fmaf(gated[g * part + c], gated[g * part + c], sum);
            sum = mlr_warp_sum(sum);
            if (lane == 0) inv[g] = 1.0f / sqrtf(sum / static_cast<float>(part) + s.eps);
        }
        __syncthreads();
    }
    T* orow = out + static_cast<size_t>(row) * ld_out;
    for (int c = threadIdx.x * V; c < total; c += blockDim.x * V) {
        float v[V];
#pragma unroll
        for (int j = 0; j < V; ++j) v[j] = gated[c + j] * inv[(c + j) / part] * (s.out_weight ? s.out_weight[c + j] : 1.0f) * s.out_scale;
        mlr_store_group<V>(orow + c, v);
    }
    mlr_grid_dependents_may_start();
}

}  // namespace

constexpr int kMaxRank = 512;

static int check_recurrence(const RecurrenceSpec& s) {
    MLR_REQUIRE(s.heads > 0 && s.qk_heads > 0 && s.heads % s.qk_heads == 0 && s.heads <= 65535,
                "linear_recurrence: %d heads cannot share %d q/k heads", s.heads, s.qk_heads);
    MLR_REQUIRE(s.dim >= 1 && s.dim <= 256 && s.vdim >= 1 && s.vdim <= 256 && !(s.dim > 128 && s.vdim > 128),
                "linear_recurrence: a state of %d x %d per head is more than a block's registers hold (256 x 128 or 128 x 256)", s.dim, s.vdim);
    MLR_REQUIRE(s.prep != 1 || (s.rot_dims >= 0 && s.rot_dims % 2 == 0 && s.rot_dims <= s.dim && (s.rot_dims == 0 || s.freq)),
                "linear_recurrence: %d rotated values do not fit a head of %d", s.rot_dims, s.dim);
    MLR_REQUIRE(s.rule >= 0 && s.rule <= 2, "linear_recurrence: no rule %d", s.rule);
    MLR_REQUIRE(s.rule != 2 || (s.skip && !s.channel_decay && s.gate_first), "linear_recurrence: the step rule goes with a skip per head and the gate before the norm");
    MLR_REQUIRE(!s.gate_first || (s.norm_parts >= 1 && (s.heads * s.vdim) % s.norm_parts == 0 && !s.gate_rank && s.eps >= 0.0f),
                "linear_recurrence: %d values of all heads cannot be normed in %d parts", s.heads * s.vdim, s.norm_parts);
    MLR_REQUIRE(!s.gate_first || sizeof(float) * (static_cast<size_t>(s.heads) * s.vdim + s.norm_parts + 4) <= 200 * 1024,
                "linear_recurrence: %d values of all heads do not fit shared memory", s.heads * s.vdim);
    if (s.channel_decay) {
        MLR_REQUIRE((s.channel_decay == 1 || (s.channel_decay == 2 && s.a_log)) && s.dt_bias && s.decay_w && s.decay_rank >= 1 &&
                        s.decay_rank <= kMaxRank, "linear_recurrence: a decay per channel needs its product (rank 1 to %d) and its constants", kMaxRank);
    } else {
        MLR_REQUIRE(s.rule == 0 ? s.decay != nullptr : (s.a_log && s.dt_bias), "linear_recurrence: the rule's constants are missing");
    }
    MLR_REQUIRE(s.gate_rank >= 0 && s.gate_rank <= kMaxRank && (!s.gate_rank || (s.gate_w && s.gate_kind && s.channel_decay && !s.norm_all)),
                "linear_recurrence: a low-rank gate (rank up to %d) goes with a decay per channel and a norm per head", kMaxRank);
    return 0;
}

namespace {
template <typename T>
void launch_readout(const RecurrenceSpec& s, const float* obuf, const T* side, int ld_side, const float* gf, T* out, int ld_out, int rows,
                    cudaStream_t stream) {
    const auto aligned = [](const void* p, size_t bytes) { return reinterpret_cast<uintptr_t>(p) % bytes == 0; };
    if (s.gate_first) {
        const int total = s.heads * s.vdim;
        const size_t shared = sizeof(float) * ((total + 3) / 4 * 4 + s.norm_parts);
        const bool four = total % 4 == 0 && aligned(obuf, 16) && aligned(out, 4 * sizeof(T)) && ld_out % 4 == 0 &&
                          (!s.gate_kind || (aligned(side + s.col_gate, 4 * sizeof(T)) && ld_side % 4 == 0));
        const auto kernel = four ? recurrence_parts_readout_kernel<T, 4> : recurrence_parts_readout_kernel<T, 1>;
        if (shared > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(shared));
        mlr_launch(kernel, dim3(rows), dim3(kReadoutThreads), shared, stream, obuf, side, ld_side, out, ld_out, s);
        return;
    }
    // Head sizes that are no multiple of 32 keep the one-kernel form's order of every sum (the same bits in both forms).
    const bool vec = s.dim % 32 == 0 && s.vdim % 4 == 0 && aligned(obuf, 16) && aligned(out, 4 * sizeof(T)) && ld_out % 4 == 0 &&
                     (!s.gate_kind || (gf ? aligned(gf, 16) : aligned(side + s.col_gate, 4 * sizeof(T)) && ld_side % 4 == 0));
    if (vec) mlr_launch((recurrence_readout_kernel<T, true>), dim3(rows), dim3(kReadoutThreads), 0, stream, obuf, side, ld_side, gf, out, ld_out, s);
    else mlr_launch((recurrence_readout_kernel<T, false>), dim3(rows), dim3(kReadoutThreads), 0, stream, obuf, side, ld_side, gf, out, ld_out, s);
}
}  // namespace

MLR_API int mlr_linear_recurrence(const RecurrenceSpec* spec, const void* proj, int ld, const void* side, int ld_side, int act_bf16, void* out, int ld_out,
                                  float* state, long long state_stride, const int* segment_info, int n_segments, int rows, float* obuf,
                                  int* status, cudaStream_t stream) {
    // `obuf` (float32 [rows, heads * vdim], or null): the kernel leaves its plain outputs there and the read-out is a
    // launch of its own over the step's `rows` rows; a description with norm_all needs it.
    (void)status;
    MLR_REQUIRE(spec, "linear_recurrence: no description");
    const RecurrenceSpec& s = *spec;
    if (check_recurrence(s)) return 1;
    MLR_REQUIRE(n_segments >= 0 && state && proj && side && out, "linear_recurrence: bad arguments");
    MLR_REQUIRE(!(s.norm_all || s.gate_first) || obuf, "linear_recurrence: a norm over all heads needs the buffer of plain outputs");
    MLR_REQUIRE(!s.gate_rank || !obuf, "linear_recurrence: plain outputs have no place for a low-rank gate");
    if (n_segments == 0) return 0;
    const int cols = s.vdim > 128 ? 8 : 4;
    const int warps = (s.vdim + cols - 1) / cols;
    const int regs = s.dim <= 32 ? 1 : s.dim <= 64 ? 2 : s.dim <= 128 ? 4 : 8;
    const bool channel = s.channel_decay != 0;
    const size_t per_token = sizeof(float) * (2 * static_cast<size_t>(s.dim) + 2 * s.vdim + 2 +
                                              (channel ? s.dim + s.decay_rank + s.gate_rank + (s.gate_rank ? s.vdim : 0) : 0));
    int batch = static_cast<int>((40 * 1024) / per_token);
    batch = batch < 1 ? 1 : (batch > 32 ? 32 : batch);
    const size_t shared = per_token * batch;
    const dim3 grid(n_segments, s.heads);
#define MLR_GO(T, R, C)                                                                                                     \
    do {                                                                                                                     \
        if (channel) MLR_GO2(T, R, C, true);                                                                                 \
        else MLR_GO2(T, R, C, false);                                                                                        \
    } while (0)
#define MLR_GO2(T, R, C, CH)                                                                                                   \
    mlr_launch((linear_recurrence_kernel<T, R, C, CH>), dim3(grid), dim3(warps * 32), shared, stream, static_cast<const T*>(proj), ld, static_cast<const T*>(side), ld_side, \
               static_cast<T*>(out), ld_out, state, state_stride, segment_info, s, batch, obuf)
#define MLR_PICK(T)                                              \
    do {                                                         \
        if (cols == 4) {                                         \
            if (regs == 1) MLR_GO(T, 1, 4);                      \
            else if (regs == 2) MLR_GO(T, 2, 4);                 \
            else if (regs == 4) MLR_GO(T, 4, 4);                 \
            else MLR_GO(T, 8, 4);                                \
        } else {                                                 \
            if (regs == 1) MLR_GO(T, 1, 8);                      \
            else if (regs == 2) MLR_GO(T, 2, 8);                 \
            else MLR_GO(T, 4, 8);                                \
        }                                                        \
    } while (0)
    if (act_bf16) MLR_PICK(__nv_bfloat16);
    else MLR_PICK(float);
#undef MLR_PICK
#undef MLR_GO
#undef MLR_GO2
    if (obuf && rows > 0) {
        if (act_bf16) launch_readout(s, obuf, static_cast<const __nv_bfloat16*>(side), ld_side, nullptr, static_cast<__nv_bfloat16*>(out), ld_out, rows, stream);
        else launch_readout(s, obuf, static_cast<const float*>(side), ld_side, nullptr, static_cast<float*>(out), ld_out, rows, stream);
    }
    return mlr_launched("linear_recurrence");
}

// The three-kernel form.  qf, kf: float32 [rows, qk_heads * dim]; gates: float32 [rows, 2 * heads] (delta and step rules; else unused);
// obuf: float32 [rows, heads * vdim].  Same results as `mlr_linear_recurrence` up to the order in which a column's sums are added
// (the same order for head sizes that are no multiple of 32).  With a decay per channel, df [rows, heads * dim] and (low-rank gate) gf
// [rows, heads * vdim] are float32 room; with `products_made` they hold the low-rank products' results already (df without the bias).
MLR_API int mlr_linear_recurrence_split(const RecurrenceSpec* spec, const void* proj, int ld, const void* side, int ld_side, int act_bf16,
                                        void* out, int ld_out, float* state, long long state_stride, const int* segment_info,
                                        int n_segments, const int* positions, int rows, float* qf, float* kf, float* gates, float* obuf,
                                        float* df, float* gf, int products_made, cudaStream_t stream) {
    MLR_REQUIRE(spec, "linear_recurrence_split: no description");
    const RecurrenceSpec& s = *spec;
    if (check_recurrence(s)) return 1;
    MLR_REQUIRE(n_segments >= 0 && rows >= 0 && state && proj && side && out && qf && kf && obuf && positions && (s.rule == 0 || gates),
                "linear_recurrence_split: bad arguments");
    MLR_REQUIRE(!s.channel_decay || (df && (!s.gate_rank || gf)), "linear_recurrence_split: a decay per channel needs its buffer, a low-rank gate too");
    if (n_segments == 0 || rows == 0) return 0;
    const int regs = s.dim <= 32 ? 1 : s.dim <= 64 ? 2 : s.dim <= 128 ? 4 : 8;
    const bool channel = s.channel_decay != 0;
    // q and k (and the channels' decays) in two stages
    // The step rule's walk takes two state columns a lane where blocks of sixteen columns would outnumber the SMs.
    const bool fixed_size = s.dim == 32 || s.dim == 64 || s.dim == 96 || s.dim == 128 || s.dim == 256;
    const int column_blocks = (s.vdim + kScanBlockCols - 1) / kScanBlockCols;
    const bool two = s.rule == 2 && fixed_size && column_blocks > 1 && static_cast<long long>(n_segments) * s.heads * column_blocks > mlr_sm_count();
    const int block_cols = kScanBlockCols * (two ? 2 : 1);
    const size_t per_token = sizeof(float) * ((channel ? 6 : 4) * static_cast<size_t>(s.dim) + 2 * block_cols + 2);
    int batch = static_cast<int>(((channel ? 84 : 44) * 1024) / per_token);
    batch = batch < 1 ? 1 : (batch > 32 ? 32 : batch);
    if (batch > 4) batch -= batch % 4;
    const size_t shared = per_token * batch + (channel ? 16 : 0);
    const dim3 grid(n_segments, s.heads, (s.vdim + block_cols - 1) / block_cols);
    const int group = s.heads * s.dim % 4 == 0 && s.heads * s.vdim % 4 == 0 ? 4 : 1;       // channels a thread of the channel kernel
    const int per_block = kChannelThreads * group;
    const dim3 channel_grid((rows + kChannelRows - 1) / kChannelRows,
                            (s.heads * s.dim + per_block - 1) / per_block + (s.gate_rank ? (s.heads * s.vdim + per_block - 1) / per_block : 0));
    const size_t channel_shared = sizeof(float) * kChannelRows * (static_cast<size_t>(s.decay_rank > s.gate_rank ? s.decay_rank : s.gate_rank) + per_block);
#define MLR_WALK(KERNEL, T, WARPS)                                                                                                     \
    do {                                                                                                                               \
        if (shared > 48 * 1024) cudaFuncSetAttribute(KERNEL, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(shared));   \
        mlr_launch((KERNEL), dim3(grid), dim3((WARPS) * 32), shared, stream, qf, kf, static_cast<const float*>(df), gates,             \
                   static_cast<const T*>(proj), ld, obuf, state, state_stride, segment_info, s, batch);                                \
    } while (0)
#define MLR_COLUMN(T, DIM, CH)                                                                                                         \
    do {                                                                                                                               \
        if (s.rule == 0) MLR_WALK((recurrence_scan16_kernel<T, DIM, 0, CH, 1>), T, kColumnWarps);                                      \
        else if (s.rule == 2 && two) MLR_WALK((recurrence_scan16_kernel<T, DIM, 2, false, 2>), T, kColumnWarps);                       \
        else if (s.rule == 2) MLR_WALK((recurrence_scan16_kernel<T, DIM, 2, false, 1>), T, kColumnWarps);                              \
        else MLR_WALK((recurrence_scan16_kernel<T, DIM, 1, CH, 1>), T, kColumnWarps);                                                  \
    } while (0)
#define MLR_SCAN(T, CH)                                                                                                                \
    do {                                                                                                                               \
        if (s.dim == 32) MLR_COLUMN(T, 32, CH);                                                                                        \
        else if (s.dim == 64) MLR_COLUMN(T, 64, CH);                                                                                   \
        else if (s.dim == 96) MLR_COLUMN(T, 96, CH);                                                                                   \
        else if (s.dim == 128) MLR_COLUMN(T, 128, CH);                                                                                 \
        else if (s.dim == 256) MLR_COLUMN(T, 256, CH);                                                                                 \
        else if (regs == 1) MLR_WALK((recurrence_scan_kernel<T, 1, CH>), T, kScanWarps);                                               \
        else if (regs == 2) MLR_WALK((recurrence_scan_kernel<T, 2, CH>), T, kScanWarps);                                               \
        else if (regs == 4) MLR_WALK((recurrence_scan_kernel<T, 4, CH>), T, kScanWarps);                                               \
        else MLR_WALK((recurrence_scan_kernel<T, 8, CH>), T, kScanWarps);                                                              \
    } while (0)
#define MLR_SPLIT(T)                                                                                                                   \
    do {                                                                                                                               \
        mlr_launch((recurrence_prepare_kernel<T>), dim3(rows), dim3(kPrepareThreads), 0, stream, static_cast<const T*>(proj), ld,      \
                   static_cast<const T*>(side), ld_side, qf, kf, gates, channel && products_made ? df : nullptr, positions, s);        \
        if (channel && products_made) {                                                                                                \
            MLR_SCAN(T, true);                                                                                                         \
        } else if (channel) {                                                                                                                 \
            if (channel_shared > 48 * 1024)                                                                                            \
                cudaFuncSetAttribute(group == 4 ? recurrence_channel_kernel<T, 4> : recurrence_channel_kernel<T, 1>,                   \
                                     cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(channel_shared));                   \
            if (group == 4) mlr_launch((recurrence_channel_kernel<T, 4>), dim3(channel_grid), dim3(kChannelThreads), channel_shared,   \
                                       stream, static_cast<const T*>(side), ld_side, df, gf, rows, s);                                 \
            else mlr_launch((recurrence_channel_kernel<T, 1>), dim3(channel_grid), dim3(kChannelThreads), channel_shared, stream,      \
                            static_cast<const T*>(side), ld_side, df, gf, rows, s);                                                    \
            MLR_SCAN(T, true);                                                                                                         \
        } else {                                                                                                                       \
            MLR_SCAN(T, false);                                                                                                        \
        }                                                                                                                              \
        launch_readout(s, obuf, static_cast<const T*>(side), ld_side, static_cast<const float*>(s.gate_rank ? gf : nullptr),           \
                       static_cast<T*>(out), ld_out, rows, stream);                                                                    \
    } while (0)
    if (act_bf16) MLR_SPLIT(__nv_bfloat16);
    else MLR_SPLIT(float);
#undef MLR_SPLIT
#undef MLR_SCAN
#undef MLR_COLUMN
#undef MLR_WALK
    return mlr_launched("linear_recurrence_split");
}
