// The description of an attention layer over a paged cache (host memory), shared by the kernels that write the cache and those that
// read it.  See attention_masked.cu for what the fields do to scores and results.
#pragma once

struct MaskedAttentionSpec {
    const float* freq;     // [rot_dims / 2] float32 on the device, or null
    const float* sinks;    // [heads] float32 on the device: the sink's score per head; null with sink set: 0
    const float* slopes;   // [heads] float32 on the device: score -= slopes[head] * distance; null: no such bias
    const float* q_weight; // the weights of a norm of q and of k that `mlr_qkv_prepare_cache` applies (float32 on the device):
    const float* k_weight; // qk_norm 1: [dim] each, shared by all heads; qk_norm 2: [heads * dim] and [kv_heads * dim]
    int heads, kv_heads, dim, vdim;
    int rot_dims, window, chunk, sink;
    int gate_kind;         // 0 none, 1 sigmoid, 2 silu, 3 sigmoid of one value per head (the gate has `heads` columns)
    int shared_kv;         // 1: a token's value is the first vdim values of its key (vdim <= dim; one vector per token is cached and a page holds keys only)
    int keep_first;        // with a window: the first keep_first positions stay visible
    int qk_norm;           // 0 none; 1 every head of q and k over its root mean square, times a weight; 2 the WHOLE projection (all heads) likewise
    int dense_cache;       // 1: `mlr_qkv_prepare_cache` serves the kernels of the plain causal attention (attention_bf16, attention_tcgen05,
                           // attention_generic) instead of this file's: it also rotates the queries in place, and writes the cache as those
                           // kernels read it ([page][K | V][kv_head][token][dim] with dim = vdim, bfloat16 rows of 64, 128 or 256 values with
                           // their 16-byte chunks swizzled by the position: `mlr_cache_col`)
    int maps;              // 2: differential attention, two attention maps a head over the same values: `heads` counts maps (map m of head h is number
                           // 2 h + m), q and k have `dim` values a map (a key's row holds those of both), the result has heads / 2 heads, each
                           //   o = a_0 - map_weight * a_1,  o / sqrt(mean(o^2) + map_eps) * out_scale
                           // 0 or 1: ordinary attention
    float scale, out_scale;
    float softcap;         // > 0: score <- softcap * tanh(score / softcap)
    float rot_mult;        // a factor on cosine and sine (`mlr_conv_rotate_cache` only)
    float map_weight, map_eps;
};

__host__ __device__ inline int attention_maps(const MaskedAttentionSpec& s) { return s.maps > 1 ? s.maps : 1; }
// Values of a cached key's row, and of a page.
__host__ __device__ inline int attention_key_row(const MaskedAttentionSpec& s) { return attention_maps(s) * s.dim; }
