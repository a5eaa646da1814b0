// csrc/seq_prep.cu — what happens between the input projection of an attention mixer and the attention itself, for mixers whose keys are
// not simply rotated: (1) sllm_seq_unit_kv — every query, key and value head divided by its root mean square (no weight), values
// optionally blended with the values an earlier layer computed for the same token, keys and values written to their page pools;
// (2) sllm_seq_latent_kv — latent attention: the low-rank row of a token is RMS-normed (with a weight) and cached together with ONE
// rotated key part that all heads share; the rotated part of every query head moves, rotated, behind that head's absorbed query.
// (3) sllm_seq_normed_rotary_kv — every query and key head RMS-normed with a weight of the head's width, then (partly) rotated by the
// position; the keys go to their pool, the values (which may be the key heads as they were before norm and rotation) to theirs;
// (4) sllm_seq_head_mix — after the attention: the heads' results mixed by a heads x heads matrix;
// (5) sllm_seq_wide_normed_rotary_kv — queries and keys RMS-normed over the whole projection (all heads of a token at once), then rotated;
// values optionally blended as in (1); the keys of a token's heads may be stored side by side, and the queries may leave as the mixed
// bf16 operand rows of attention whose scores are mixed over the heads before the softmax;
// (6) sllm_seq_angles — cos and sin of every token's position times every frequency, once per step for all layers that turn alike.
// (7) sllm_seq_conv_rotary_kv — every query, key and value head through a short causal convolution (optional), queries and keys then turned by
// the step's angles and (optionally) divided by their root mean square; keys and values written to their pools, the convolution's last
// inputs to their ring in steps of single tokens.
// All arithmetic is fp32 (angles in double); the pools hold fp32 or bf16.
#include "seq_common.cuh"

namespace sllm {

// grid (T, ceil(items / 4)), 4 warps: warp = one head of q, k or v of one token
template <typename KV>
__global__ void seq_unit_kv_kernel(sllm_seq_batch b, float* __restrict__ q, int ldq, int heads, int dk, const float* __restrict__ k, int ldk, int kv_heads,
                                   const float* __restrict__ v, int ldv, int dv, float eps, int unit, float* __restrict__ v_shared, int share, float lambda,
                                   float q_temp_coef, int q_temp_every, KV* __restrict__ k_pool, KV* __restrict__ v_pool) {
    const int t = blockIdx.x, item = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (item >= heads + 2 * kv_heads) return;
    const int pos = b.tok_pos[t], slot = b.tok_slot[t];
    const int page = b.block_table[(size_t)slot * b.max_pages + pos / b.page_len], in_page = pos % b.page_len;
    if (item < heads) {                                  // a query head, in place
        // query temperature: queries grow with the logarithm of the position, in steps of q_temp_every positions
        const float temp = q_temp_every > 0 ? 1.0f + q_temp_coef * logf((float)((pos + 1) / q_temp_every) + 1.0f) : 1.0f;
        if (!(unit & 1) && temp == 1.0f) return;
        float* row = q + (size_t)t * ldq + (size_t)item * dk;
        float inv = temp;
        if (unit & 1) {
            float ss = 0.0f;
            for (int j = lane; j < dk; j += 32) ss = fmaf(row[j], row[j], ss);
            inv = temp / sqrtf(warp_sum(ss) / (float)dk + eps);
        }
        for (int j = lane; j < dk; j += 32) row[j] *= inv;
    } else if (item < heads + kv_heads) {                // a key head -> pool
        const int g = item - heads;
        const float* row = k + (size_t)t * ldk + (size_t)g * dk;
        float inv = 1.0f;
        if (unit & 2) {
            float ss = 0.0f;
            for (int j = lane; j < dk; j += 32) ss = fmaf(row[j], row[j], ss);
            inv = 1.0f / sqrtf(warp_sum(ss) / (float)dk + eps);
        }
        const size_t dst = seq_pool_row(page, kv_heads, g, b.page_len, in_page, dk);
        for (int j = lane; j < dk; j += 32) seq_st(k_pool, dst + j, row[j] * inv);
    } else {                                             // a value head -> (blend) -> pool
        const int g = item - heads - kv_heads;
        const float* row = v + (size_t)t * ldv + (size_t)g * dv;
        float inv = 1.0f;
        if (unit & 4) {
            float ss = 0.0f;
            for (int j = lane; j < dv; j += 32) ss = fmaf(row[j], row[j], ss);
            inv = 1.0f / sqrtf(warp_sum(ss) / (float)dv + eps);
        }
        const size_t dst = seq_pool_row(page, kv_heads, g, b.page_len, in_page, dv);
        float* sh = v_shared ? v_shared + ((size_t)t * kv_heads + g) * dv : nullptr;
        for (int j = lane; j < dv; j += 32) {
            float val = row[j] * inv;
            if (share == 1) sh[j] = val;
            else if (share == 2) val = (1.0f - lambda) * val + lambda * sh[j];
            seq_st(v_pool, dst + j, val);
        }
    }
}

// one CTA per token
template <typename KV>
__global__ void seq_latent_kv_kernel(sllm_seq_batch b, const float* __restrict__ q, int ldq, int heads, int dn, int dr, const float* __restrict__ low, int ldlow,
                                     int rank, const float* __restrict__ norm_w, float eps, const double* __restrict__ freq, int n_freq, float magnitude,
                                     float* __restrict__ q_out, int ldqo, KV* __restrict__ pool) {
    __shared__ float red[33];
    const int t = blockIdx.x, pos = b.tok_pos[t], slot = b.tok_slot[t];
    const int page = b.block_table[(size_t)slot * b.max_pages + pos / b.page_len], in_page = pos % b.page_len;
    const float* lr = low ? low + (size_t)t * ldlow : nullptr;   // no low-rank row: the layer reads another layer's cache, only its queries turn
    const size_t dst = seq_pool_row(page, 1, 0, b.page_len, in_page, rank + dr);
    const int items = low ? heads + 1 : heads;
    if (low) {
        float ss = 0.0f;
        for (int j = threadIdx.x; j < rank; j += blockDim.x) ss = fmaf(lr[j], lr[j], ss);
        ss = block_sum(ss, red);
        const float inv = 1.0f / sqrtf(ss / (float)rank + eps);
        for (int j = threadIdx.x; j < rank; j += blockDim.x) seq_st(pool, dst + j, (lr[j] * inv) * norm_w[j]);
    }
    // rotated pairs: item 0 .. heads-1 = the query heads, item heads = the shared key part; the first 2 * n_freq dimensions turn
    for (int i = threadIdx.x; i < items * n_freq; i += blockDim.x) {
        const int h = i / n_freq, mi = i % n_freq;
        float sn, cs;
        seq_angle(pos, freq[mi], &sn, &cs);
        sn *= magnitude;
        cs *= magnitude;
        const float* src = h < heads ? q + (size_t)t * ldq + (size_t)h * (dn + dr) + dn : lr + rank;
        const float u = src[2 * mi], w = src[2 * mi + 1];
        const float a = u * cs - w * sn, c = w * cs + u * sn;
        if (h < heads) {
            float* o = q_out + (size_t)t * ldqo + (size_t)h * (rank + dr) + rank;
            o[2 * mi] = a;
            o[2 * mi + 1] = c;
        } else {
            seq_st(pool, dst + rank + 2 * mi, a);
            seq_st(pool, dst + rank + 2 * mi + 1, c);
        }
    }
    const int rest = dr - 2 * n_freq;                     // dimensions of the rotated part beyond the rotary ones pass unchanged
    for (int i = threadIdx.x; i < items * rest; i += blockDim.x) {
        const int h = i / rest, j = 2 * n_freq + i % rest;
        if (h < heads) q_out[(size_t)t * ldqo + (size_t)h * (rank + dr) + rank + j] = q[(size_t)t * ldq + (size_t)h * (dn + dr) + dn + j];
        else seq_st(pool, dst + rank + j, lr[rank + j]);
    }
}

// grid (T, ceil(items / 4)), 4 warps: warp = one query head (normed and rotated in place), one key head (normed, rotated -> pool) or one
// value head (-> pool as it is); the head's row sits in shared memory while its pairs turn
template <typename KV>
__global__ void seq_normed_rotary_kv_kernel(sllm_seq_batch b, float* __restrict__ q, int ldq, int heads, int dk, const float* __restrict__ k, int ldk, int kv_heads,
                                            const float* __restrict__ v, int ldv, int dv, const float* __restrict__ q_w, const float* __restrict__ k_w, float eps,
                                            const double* __restrict__ freq, int n_freq, int layout, KV* __restrict__ k_pool, KV* __restrict__ v_pool) {
    extern __shared__ float nr_sm[];                     // [4][dk]
    const int t = blockIdx.x, item = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (item >= heads + 2 * kv_heads) return;
    const int pos = b.tok_pos[t], slot = b.tok_slot[t];
    const int page = b.block_table[(size_t)slot * b.max_pages + pos / b.page_len], in_page = pos % b.page_len;
    if (item >= heads + kv_heads) {                      // a value head
        const int g = item - heads - kv_heads;
        const float* row = v + (size_t)t * ldv + (size_t)g * dv;
        const size_t dst = seq_pool_row(page, kv_heads, g, b.page_len, in_page, dv);
        for (int j = lane; j < dv; j += 32) seq_st(v_pool, dst + j, row[j]);
        return;
    }
    const bool is_q = item < heads;
    const int g = is_q ? item : item - heads;
    const float* row = is_q ? q + (size_t)t * ldq + (size_t)g * dk : k + (size_t)t * ldk + (size_t)g * dk;
    const float* w = is_q ? q_w : k_w;
    float* s_row = nr_sm + (threadIdx.x >> 5) * dk;
    float ss = 0.0f;
    for (int j = lane; j < dk; j += 32) {
        const float x = row[j];
        s_row[j] = x;
        ss = fmaf(x, x, ss);
    }
    const float inv = w ? 1.0f / sqrtf(warp_sum(ss) / (float)dk + eps) : 1.0f;
    __syncwarp();
    const int half = n_freq;                             // layout 1 pairs dimension i with i + n_freq
    const size_t dst = is_q ? 0 : seq_pool_row(page, kv_heads, g, b.page_len, in_page, dk);
    float* qrow = q + (size_t)t * ldq + (size_t)g * dk;
    auto put = [&](int j, float val) {
        if (is_q) qrow[j] = val;
        else seq_st(k_pool, dst + j, val);
    };
    for (int i = lane; i < n_freq; i += 32) {
        const int ia = layout == 0 ? 2 * i : i, ib = layout == 0 ? 2 * i + 1 : i + half;
        const float u = s_row[ia] * inv * (w ? w[ia] : 1.0f), x = s_row[ib] * inv * (w ? w[ib] : 1.0f);
        float sn, cs;
        seq_angle(pos, freq[i], &sn, &cs);
        put(ia, u * cs - x * sn);
        put(ib, x * cs + u * sn);
    }
    for (int j = 2 * n_freq + lane; j < dk; j += 32) put(j, s_row[j] * inv * (w ? w[j] : 1.0f));
}

// four consecutive elements of a pool
__device__ __forceinline__ void seq_st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void seq_st4(uint16_t* p, float4 v) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
}

// thread = (token, frequency)
__global__ void seq_angles_kernel(sllm_seq_batch b, const double* __restrict__ freq, int n_freq, float2* __restrict__ out) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= b.T * n_freq) return;
    float sn, cs;
    seq_angle(b.tok_pos[i / n_freq], freq[i % n_freq], &sn, &cs);
    out[i] = make_float2(cs, sn);
}

// grid (T, 2): CTA y = 0 takes a token's queries, CTA y = 1 its keys and values. The whole row sits in shared memory (its root mean square
// is over all heads); the token's angles come from the step's table.
constexpr int kMixGroup = 8;   // query heads of a key head whose values a thread holds at once while it mixes

template <typename KV>
__global__ void __launch_bounds__(256) seq_wide_normed_rotary_kv_kernel(sllm_seq_batch b, float* __restrict__ q, int ldq, int heads, int dk, const float* __restrict__ k,
                                                                        int ldk, int kv_heads, const float* __restrict__ v, int ldv, int dv, const float* __restrict__ q_w,
                                                                        const float* __restrict__ k_w, float eps, const float2* __restrict__ angles, int n_freq, int layout,
                                                                        float* __restrict__ v_shared, int share, float lambda, const float* __restrict__ talk,
                                                                        uint16_t* __restrict__ q_mixed, int k_joint, KV* __restrict__ k_pool, KV* __restrict__ v_pool,
                                                                        int vec) {
    extern __shared__ __align__(16) float wr_sm[];       // the row, and for the mix talk [heads][heads]
    __shared__ float red[33];
    const int t = blockIdx.x, pos = b.tok_pos[t], slot = b.tok_slot[t];
    const bool is_q = blockIdx.y == 0;
    const int n_heads = is_q ? heads : kv_heads, n = n_heads * dk, group = heads / kv_heads;
    float* s_row = wr_sm;
    float* s_talk = wr_sm + ((heads * dk + 3) & ~3);
    const float2* turn = angles + (size_t)t * n_freq;
    float* row = is_q ? q + (size_t)t * ldq : nullptr;
    const float* src = is_q ? row : k + (size_t)t * ldk;
    const float* w = is_q ? q_w : k_w;
    if (is_q && q_mixed)
        for (int i = threadIdx.x; i < heads * heads; i += blockDim.x) s_talk[i] = talk[i];
    float ss = 0.0f;
    if (vec) {                                           // four columns at a time, every thread its own columns in both passes
#pragma unroll 4
        for (int j = 4 * threadIdx.x; j < n; j += 4 * blockDim.x) {
            const float4 x = *reinterpret_cast<const float4*>(src + j);
            *reinterpret_cast<float4*>(s_row + j) = x;
            ss = fmaf(x.x, x.x, fmaf(x.y, x.y, fmaf(x.z, x.z, fmaf(x.w, x.w, ss))));
        }
    } else {
        for (int j = threadIdx.x; j < n; j += blockDim.x) {
            const float x = src[j];
            s_row[j] = x;
            ss = fmaf(x, x, ss);
        }
    }
    ss = block_sum(ss, red);
    if (w) {
        const float inv = 1.0f / sqrtf(ss / (float)n + eps);
        if (vec) {
#pragma unroll 4
            for (int j = 4 * threadIdx.x; j < n; j += 4 * blockDim.x) {
                const float4 x = *reinterpret_cast<const float4*>(s_row + j), g = *reinterpret_cast<const float4*>(w + j);
                *reinterpret_cast<float4*>(s_row + j) = make_float4((x.x * inv) * g.x, (x.y * inv) * g.y, (x.z * inv) * g.z, (x.w * inv) * g.w);
            }
        } else {
            for (int j = threadIdx.x; j < n; j += blockDim.x) s_row[j] = (s_row[j] * inv) * w[j];
        }
        __syncthreads();
    }
    for (int i = threadIdx.x; i < n_heads * n_freq; i += blockDim.x) {
        const int h = i / n_freq, mi = i % n_freq;
        const int ia = h * dk + (layout == 0 ? 2 * mi : mi), ib = h * dk + (layout == 0 ? 2 * mi + 1 : mi + n_freq);
        const float2 a = turn[mi];
        const float u = s_row[ia], x = s_row[ib];
        s_row[ia] = u * a.x - x * a.y;
        s_row[ib] = x * a.x + u * a.y;
    }
    __syncthreads();
    if (!is_q) {
        const int page = b.block_table[(size_t)slot * b.max_pages + pos / b.page_len], in_page = pos % b.page_len;
        if (vec) {
            for (int j = 4 * threadIdx.x; j < n; j += 4 * blockDim.x) {
                const size_t dst = k_joint ? ((size_t)page * b.page_len + in_page) * n + j : seq_pool_row(page, kv_heads, j / dk, b.page_len, in_page, dk) + j % dk;
                seq_st4(k_pool + dst, *reinterpret_cast<const float4*>(s_row + j));
            }
            for (int j = 4 * threadIdx.x; j < kv_heads * dv; j += 4 * blockDim.x) {
                float4 val = *reinterpret_cast<const float4*>(v + (size_t)t * ldv + j);
                float4* sh = share ? reinterpret_cast<float4*>(v_shared + (size_t)t * kv_heads * dv + j) : nullptr;
                if (share == 1) {
                    *sh = val;
                } else if (share == 2) {
                    const float4 first = *sh;
                    const float mine = 1.0f - lambda;
                    val = make_float4(mine * val.x + lambda * first.x, mine * val.y + lambda * first.y, mine * val.z + lambda * first.z, mine * val.w + lambda * first.w);
                }
                seq_st4(v_pool + seq_pool_row(page, kv_heads, j / dv, b.page_len, in_page, dv) + j % dv, val);
            }
            return;
        }
        if (k_joint) {
            const size_t dst = ((size_t)page * b.page_len + in_page) * n;
            for (int j = threadIdx.x; j < n; j += blockDim.x) seq_st(k_pool, dst + j, s_row[j]);
        } else {
            for (int j = threadIdx.x; j < n; j += blockDim.x) seq_st(k_pool, seq_pool_row(page, kv_heads, j / dk, b.page_len, in_page, dk) + j % dk, s_row[j]);
        }
        for (int j = threadIdx.x; j < kv_heads * dv; j += blockDim.x) {
            float val = v[(size_t)t * ldv + j];
            if (share == 1) v_shared[(size_t)t * kv_heads * dv + j] = val;
            else if (share == 2) val = (1.0f - lambda) * val + lambda * v_shared[(size_t)t * kv_heads * dv + j];
            seq_st(v_pool, seq_pool_row(page, kv_heads, j / dv, b.page_len, in_page, dv) + j % dv, val);
        }
        return;
    }
    if (!q_mixed) {
        for (int j = threadIdx.x; j < n; j += blockDim.x) row[j] = s_row[j];
        return;
    }
    // part u of mixed head h: sum over the query heads g of key head u of talk[h][g] * q_g
    const int wide = kv_heads * dk;
    uint16_t* out = q_mixed + (size_t)t * heads * wide;
    if (dk % 4 == 0 && group <= kMixGroup) {             // a thread keeps four columns of a group's queries and walks over the mixed heads
        const int quads = wide / 4, lanes = max(1, (int)blockDim.x / quads);
        for (int i = threadIdx.x; i < quads * lanes; i += blockDim.x) {
            const int qd = i % quads, u = 4 * qd / dk, c = 4 * qd % dk;
            float4 x[kMixGroup];
#pragma unroll
            for (int g = 0; g < kMixGroup; ++g)
                if (g < group) x[g] = *reinterpret_cast<const float4*>(s_row + (size_t)(u * group + g) * dk + c);
            for (int h = i / quads; h < heads; h += lanes) {
                float4 acc = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                const float* tr = s_talk + h * heads + u * group;
                __align__(16) float tws[kMixGroup];
                if (group % 4 == 0) {                    // (then heads is a multiple of four, and so is the row's start)
#pragma unroll
                    for (int g = 0; g < kMixGroup; g += 4)
                        if (g < group) *reinterpret_cast<float4*>(tws + g) = *reinterpret_cast<const float4*>(tr + g);
                } else {
#pragma unroll
                    for (int g = 0; g < kMixGroup; ++g)
                        if (g < group) tws[g] = tr[g];
                }
#pragma unroll
                for (int g = 0; g < kMixGroup; ++g) {
                    if (g < group) {
                        const float tw = tws[g];
                        acc.x = fmaf(tw, x[g].x, acc.x);
                        acc.y = fmaf(tw, x[g].y, acc.y);
                        acc.z = fmaf(tw, x[g].z, acc.z);
                        acc.w = fmaf(tw, x[g].w, acc.w);
                    }
                }
                seq_st4(out + (size_t)h * wide + 4 * qd, acc);
            }
        }
        return;
    }
    for (int i = threadIdx.x; i < heads * wide; i += blockDim.x) {
        const int h = i / wide, j = i % wide, u = j / dk, c = j % dk;
        float acc = 0.0f;
        for (int g = 0; g < group; ++g) acc = fmaf(s_talk[h * heads + u * group + g], s_row[(size_t)(u * group + g) * dk + c], acc);
        out[i] = f32_to_bf16_bits(acc);
    }
}

struct ConvRotaryArgs {
    sllm_seq_batch b;
    const float *q, *k, *v; int ldq, ldk, ldv;           // projections: q [heads][dk], k [kv_heads][dk], v [kv_heads][dv] per token
    int heads, kv_heads, dk, dv;
    const float* conv_w; int taps; float* ring;          // [taps][channels] (oldest first), channels = q, k, v in this order; ring [slots][taps-1][channels]; NULL = no convolution
    int store_ring;                                      // every portion is one token: the token's inputs go to the ring here
    const float2* angles; int n_freq, layout;            // (cos, sin) [T][n_freq]
    int unit; float eps;                                 // 1: queries and keys divided by their root mean square after they turned
    float* q_out; int ldqo;                              // may be q itself when there is no convolution
    void *k_pool, *v_pool;
    int tile, vec;                                       // tokens a warp walks; 16-byte accesses
};

// grid (ceil(T / tile), ceil(items / 4)), 4 warps: warp = one head of q, k or v over a tile of tokens; the head's row of the token at hand
// sits in shared memory while its pairs turn
template <typename KV>
__global__ void __launch_bounds__(128) seq_conv_rotary_kv_kernel(ConvRotaryArgs p) {
    extern __shared__ __align__(16) float cr_sm[];       // [4][max(dk, dv)]
    const sllm_seq_batch& b = p.b;
    const int item = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (item >= p.heads + 2 * p.kv_heads) return;
    const bool is_q = item < p.heads, is_v = item >= p.heads + p.kv_heads;
    const int g = is_q ? item : (is_v ? item - p.heads - p.kv_heads : item - p.heads), width = is_v ? p.dv : p.dk;
    const float* src = (is_q ? p.q : (is_v ? p.v : p.k)) + (size_t)g * width;
    const int ld = is_q ? p.ldq : (is_v ? p.ldv : p.ldk);
    const int channels = (p.heads + p.kv_heads) * p.dk + p.kv_heads * p.dv;
    const int ch0 = is_q ? g * p.dk : (is_v ? (p.heads + p.kv_heads) * p.dk + g * p.dv : (p.heads + g) * p.dk);   // the head's first channel of the convolution
    float* row = cr_sm + (threadIdx.x >> 5) * ((max(p.dk, p.dv) + 3) & ~3);
    const int t1 = min(b.T, (int)(blockIdx.x + 1) * p.tile);
    for (int t = blockIdx.x * p.tile; t < t1; ++t) {
        const int pos = b.tok_pos[t], slot = b.tok_slot[t];
        const int page = b.block_table[(size_t)slot * b.max_pages + pos / b.page_len], in_page = pos % b.page_len;
        // the input row `back` positions before the token: a row of this step, a row of the ring, or (before the start) nothing
        auto earlier = [&](int back) -> const float* {
            if (pos - back < 0) return nullptr;
            if (back == 0 || (t - back >= 0 && b.tok_slot[t - back] == slot)) return src + (size_t)(t - back) * ld;
            return p.ring + ((size_t)slot * (p.taps - 1) + (pos - back) % (p.taps - 1)) * channels + ch0;
        };
        float* keep = p.store_ring ? p.ring + ((size_t)slot * (p.taps - 1) + pos % (p.taps - 1)) * channels + ch0 : nullptr;
        float ss = 0.0f;
        if (p.vec) {
            for (int j = 4 * lane; j < width; j += 128) {
                const float4 own = *reinterpret_cast<const float4*>(src + (size_t)t * ld + j);
                float4 a = own;
                if (p.conv_w) {
                    const float4 w0 = *reinterpret_cast<const float4*>(p.conv_w + (size_t)(p.taps - 1) * channels + ch0 + j);
                    a = make_float4(w0.x * own.x, w0.y * own.y, w0.z * own.z, w0.w * own.w);
                    for (int back = 1; back < p.taps; ++back) {
                        const float* e = earlier(back);
                        if (!e) break;
                        const float4 x = *reinterpret_cast<const float4*>(e + j), w = *reinterpret_cast<const float4*>(p.conv_w + (size_t)(p.taps - 1 - back) * channels + ch0 + j);
                        a = make_float4(fmaf(w.x, x.x, a.x), fmaf(w.y, x.y, a.y), fmaf(w.z, x.z, a.z), fmaf(w.w, x.w, a.w));
                    }
                    if (keep) *reinterpret_cast<float4*>(keep + j) = own;      // the oldest row of the ring, read above by this thread
                }
                *reinterpret_cast<float4*>(row + j) = a;
                ss = fmaf(a.x, a.x, fmaf(a.y, a.y, fmaf(a.z, a.z, fmaf(a.w, a.w, ss))));
            }
        } else {
            for (int j = lane; j < width; j += 32) {
                const float own = src[(size_t)t * ld + j];
                float a = own;
                if (p.conv_w) {
                    a = p.conv_w[(size_t)(p.taps - 1) * channels + ch0 + j] * own;
                    for (int back = 1; back < p.taps; ++back) {
                        const float* e = earlier(back);
                        if (!e) break;
                        a = fmaf(p.conv_w[(size_t)(p.taps - 1 - back) * channels + ch0 + j], e[j], a);
                    }
                    if (keep) keep[j] = own;
                }
                row[j] = a;
                ss = fmaf(a, a, ss);
            }
        }
        __syncwarp();
        if (!is_v && p.n_freq) {
            for (int i = lane; i < p.n_freq; i += 32) {
                const int ia = p.layout == 0 ? 2 * i : i, ib = p.layout == 0 ? 2 * i + 1 : i + p.n_freq;
                const float2 a = p.angles[(size_t)t * p.n_freq + i];
                const float u = row[ia], w = row[ib];
                row[ia] = u * a.x - w * a.y;
                row[ib] = w * a.x + u * a.y;
            }
            __syncwarp();
        }
        float inv = 1.0f;
        if (!is_v && p.unit) {
            if (p.n_freq) {                              // of the turned row, as defined
                ss = 0.0f;
                for (int j = lane; j < width; j += 32) ss = fmaf(row[j], row[j], ss);
            }
            inv = 1.0f / sqrtf(warp_sum(ss) / (float)width + p.eps);
        }
        KV* pool = reinterpret_cast<KV*>(is_v ? p.v_pool : p.k_pool);
        const size_t dst = is_q ? 0 : seq_pool_row(page, p.kv_heads, g, b.page_len, in_page, width);
        float* qrow = p.q_out + (size_t)t * p.ldqo + (size_t)g * width;
        if (p.vec) {
            for (int j = 4 * lane; j < width; j += 128) {
                const float4 a = *reinterpret_cast<const float4*>(row + j);
                const float4 o = make_float4(a.x * inv, a.y * inv, a.z * inv, a.w * inv);
                if (is_q) *reinterpret_cast<float4*>(qrow + j) = o;
                else seq_st4(pool + dst + j, o);
            }
        } else {
            for (int j = lane; j < width; j += 32) {
                if (is_q) qrow[j] = row[j] * inv;
                else seq_st(pool, dst + j, row[j] * inv);
            }
        }
        __syncwarp();                                    // the row is free for the next token
    }
}

// The same for heads of up to 128 channels in interleaved pairs, 16-byte rows and up to four taps: a lane keeps four channels of its head in
// registers — the weights over the tile of tokens, the pairs that turn — and nothing passes through shared memory.
template <typename KV, int TAPS>   // TAPS 0: no convolution
__global__ void __launch_bounds__(128) seq_conv_rotary_kv_row_kernel(ConvRotaryArgs p) {
    const sllm_seq_batch& b = p.b;
    const int item = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (item >= p.heads + 2 * p.kv_heads) return;
    const bool is_q = item < p.heads, is_v = item >= p.heads + p.kv_heads;
    const int g = is_q ? item : (is_v ? item - p.heads - p.kv_heads : item - p.heads), width = is_v ? p.dv : p.dk;
    const int ld = is_q ? p.ldq : (is_v ? p.ldv : p.ldk), j = 4 * lane;
    const float* src = (is_q ? p.q : (is_v ? p.v : p.k)) + (size_t)g * width + j;
    const int channels = (p.heads + p.kv_heads) * p.dk + p.kv_heads * p.dv;
    const int ch = (is_q ? g * p.dk : (is_v ? (p.heads + p.kv_heads) * p.dk + g * p.dv : (p.heads + g) * p.dk)) + j;   // of the convolution
    const bool live = j < width;
    const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    float4 w[TAPS > 0 ? TAPS : 1];                                 // [back]
#pragma unroll
    for (int back = 0; back < TAPS; ++back) w[back] = live ? *reinterpret_cast<const float4*>(p.conv_w + (size_t)(TAPS - 1 - back) * channels + ch) : zero;
    KV* pool = reinterpret_cast<KV*>(is_v ? p.v_pool : p.k_pool);
    const bool turns = !is_v && lane < (p.n_freq + 1) / 2;         // this lane holds pairs 2 * lane and 2 * lane + 1
    const int t0 = blockIdx.x * p.tile, t1 = min(b.T, t0 + p.tile);
    for (int t = t0; t < t1; ++t) {
        const float4 own = live ? *reinterpret_cast<const float4*>(src + (size_t)t * ld) : zero;
        const int pos = b.tok_pos[t], slot = b.tok_slot[t];
        float4 a = own;
        if (TAPS > 0) {
            a = make_float4(w[0].x * own.x, w[0].y * own.y, w[0].z * own.z, w[0].w * own.w);
#pragma unroll
            for (int back = 1; back < TAPS; ++back) {              // the rows before it: this step's (near in the cache), the ring's, or nothing
                if (live && pos - back >= 0) {
                    const float4 x = (t - back >= 0 && b.tok_slot[t - back] == slot)
                                         ? *reinterpret_cast<const float4*>(src + (size_t)(t - back) * ld)
                                         : *reinterpret_cast<const float4*>(p.ring + ((size_t)slot * (TAPS - 1) + (pos - back) % (TAPS - 1)) * channels + ch);
                    a = make_float4(fmaf(w[back].x, x.x, a.x), fmaf(w[back].y, x.y, a.y), fmaf(w[back].z, x.z, a.z), fmaf(w[back].w, x.w, a.w));
                }
            }
            // single tokens: the oldest row of the ring, read above by this thread
            if (TAPS > 1 && p.store_ring && live) *reinterpret_cast<float4*>(p.ring + ((size_t)slot * (TAPS - 1) + pos % (TAPS - 1)) * channels + ch) = own;
        }
        if (turns) {
            const float2 r0 = p.angles[(size_t)t * p.n_freq + 2 * lane];
            const float u0 = a.x, v0 = a.y;
            a.x = u0 * r0.x - v0 * r0.y;
            a.y = v0 * r0.x + u0 * r0.y;
            if (2 * lane + 1 < p.n_freq) {
                const float2 r1 = p.angles[(size_t)t * p.n_freq + 2 * lane + 1];
                const float u1 = a.z, v1 = a.w;
                a.z = u1 * r1.x - v1 * r1.y;
                a.w = v1 * r1.x + u1 * r1.y;
            }
        }
        if (!is_v && p.unit) {
            const float ss = warp_sum(live ? fmaf(a.x, a.x, fmaf(a.y, a.y, fmaf(a.z, a.z, a.w * a.w))) : 0.0f);
            const float inv = 1.0f / sqrtf(ss / (float)width + p.eps);
            a = make_float4(a.x * inv, a.y * inv, a.z * inv, a.w * inv);
        }
        if (!live) continue;
        if (is_q) {
            *reinterpret_cast<float4*>(p.q_out + (size_t)t * p.ldqo + (size_t)g * width + j) = a;
        } else {
            const int page = b.block_table[(size_t)slot * b.max_pages + pos / b.page_len];
            seq_st4(pool + seq_pool_row(page, p.kv_heads, g, b.page_len, pos % b.page_len, width) + j, a);
        }
    }
}

// thread = (token, head, column): out[t][h][c] = sum_g mix[h][g] * in[t][(h / group) * heads + g][c], group = heads / kv_heads: `in` holds,
// for every key/value head, the result of EVERY query head's weights on that head's values
__global__ void seq_head_mix_kernel(const float* __restrict__ in, int ldi, const float* __restrict__ mix, int heads, int kv_heads, int dv,
                                    float* __restrict__ out, int ldo, uint16_t* __restrict__ out16, int T) {
    extern __shared__ float hm_sm[];                     // [heads][heads]
    for (int i = threadIdx.x; i < heads * heads; i += blockDim.x) hm_sm[i] = mix[i];
    __syncthreads();
    const int t = blockIdx.x, group = heads / kv_heads;
    const float* row = in + (size_t)t * ldi;
    for (int i = threadIdx.x; i < heads * dv; i += blockDim.x) {
        const int h = i / dv, c = i % dv;
        const float* src = row + (size_t)(h / group) * heads * dv + c;
        float acc = 0.0f;
        for (int g = 0; g < heads; ++g) acc = fmaf(hm_sm[h * heads + g], src[(size_t)g * dv], acc);
        if (out) out[(size_t)t * ldo + i] = acc;
        if (out16) out16[(size_t)t * heads * dv + i] = f32_to_bf16_bits(acc);
    }
}

}  // namespace sllm

using namespace sllm;

extern "C" {

int sllm_seq_unit_kv(const sllm_seq_batch* b, float* q, int32_t ldq, int32_t heads, int32_t dk, const float* k, int32_t ldk, int32_t kv_heads,
                     const float* v, int32_t ldv, int32_t dv, float eps, int32_t unit, float* v_shared, int32_t share, float lambda, void* k_pool,
                     void* v_pool, int32_t kv_dtype, float q_temp_coef, int32_t q_temp_every, sllm_stream_t stream) {
    SLLM_REQUIRE(b && b->T > 0 && b->tok_slot && b->tok_pos && b->block_table, SLLM_EINVAL, "seq_unit_kv: incomplete batch description");
    SLLM_REQUIRE(q && k && v && k_pool && v_pool && heads > 0 && kv_heads > 0 && dk > 0 && dv > 0, SLLM_EINVAL, "seq_unit_kv: bad argument");
    SLLM_REQUIRE(share >= 0 && share <= 2 && (share == 0 || v_shared), SLLM_EINVAL, "seq_unit_kv: share 0 (none), 1 (write) or 2 (blend) with a buffer");
    SLLM_REQUIRE(kv_dtype == SLLM_F32 || kv_dtype == SLLM_BF16, SLLM_ENOTSUP, "seq_unit_kv: fp32 or bf16 pools");
    const dim3 grid(b->T, (heads + 2 * kv_heads + 3) / 4);
    if (kv_dtype == SLLM_F32)
        seq_unit_kv_kernel<float><<<grid, 128, 0, as_stream(stream)>>>(*b, q, ldq, heads, dk, k, ldk, kv_heads, v, ldv, dv, eps, unit, v_shared, share, lambda,
                                                                       q_temp_coef, q_temp_every, (float*)k_pool, (float*)v_pool);
    else
        seq_unit_kv_kernel<uint16_t><<<grid, 128, 0, as_stream(stream)>>>(*b, q, ldq, heads, dk, k, ldk, kv_heads, v, ldv, dv, eps, unit, v_shared, share, lambda,
                                                                          q_temp_coef, q_temp_every, (uint16_t*)k_pool, (uint16_t*)v_pool);
    ++g_launches;
    SLLM_LAUNCH_CHECK();
    return SLLM_OK;
}

int sllm_seq_latent_kv(const sllm_seq_batch* b, const float* q, int32_t ldq, int32_t heads, int32_t dn, int32_t dr, const float* low, int32_t ldlow,
                       int32_t rank, const float* norm_w, float eps, const double* freq, int32_t n_freq, float* q_out, int32_t ldqo, void* pool,
                       int32_t kv_dtype, float magnitude, sllm_stream_t stream) {
    SLLM_REQUIRE(b && b->T > 0 && b->tok_slot && b->tok_pos && b->block_table, SLLM_EINVAL, "seq_latent_kv: incomplete batch description");
    SLLM_REQUIRE(q && q_out && (!low || (norm_w && pool)) && heads > 0 && dn >= 0 && dr >= 0 && rank > 0, SLLM_EINVAL, "seq_latent_kv: bad argument");
    SLLM_REQUIRE(n_freq >= 0 && 2 * n_freq <= dr && (n_freq == 0 || freq), SLLM_EINVAL, "seq_latent_kv: %d rotary pairs do not fit %d dimensions", n_freq, dr);
    SLLM_REQUIRE(kv_dtype == SLLM_F32 || kv_dtype == SLLM_BF16, SLLM_ENOTSUP, "seq_latent_kv: fp32 or bf16 pools");
    const int threads = rank >= 512 ? 256 : 128;
    if (kv_dtype == SLLM_F32)
        seq_latent_kv_kernel<float><<<b->T, threads, 0, as_stream(stream)>>>(*b, q, ldq, heads, dn, dr, low, ldlow, rank, norm_w, eps, freq, n_freq, magnitude, q_out, ldqo,
                                                                             (float*)pool);
    else
        seq_latent_kv_kernel<uint16_t><<<b->T, threads, 0, as_stream(stream)>>>(*b, q, ldq, heads, dn, dr, low, ldlow, rank, norm_w, eps, freq, n_freq, magnitude, q_out,
                                                                                ldqo, (uint16_t*)pool);
    ++g_launches;
    SLLM_LAUNCH_CHECK();
    return SLLM_OK;
}

int sllm_seq_normed_rotary_kv(const sllm_seq_batch* b, float* q, int32_t ldq, int32_t heads, int32_t dk, const float* k, int32_t ldk, int32_t kv_heads,
                              const float* v, int32_t ldv, int32_t dv, const float* q_norm_w, const float* k_norm_w, float eps, const double* freq,
                              int32_t n_freq, int32_t layout, void* k_pool, void* v_pool, int32_t kv_dtype, sllm_stream_t stream) {
    SLLM_REQUIRE(b && b->T > 0 && b->tok_slot && b->tok_pos && b->block_table, SLLM_EINVAL, "seq_normed_rotary_kv: incomplete batch description");
    SLLM_REQUIRE(q && k && v && k_pool && v_pool && heads > 0 && kv_heads > 0 && dk > 0 && dv > 0, SLLM_EINVAL, "seq_normed_rotary_kv: bad argument");
    SLLM_REQUIRE(n_freq >= 0 && 2 * n_freq <= dk && (n_freq == 0 || freq), SLLM_EINVAL, "seq_normed_rotary_kv: %d rotary pairs do not fit %d dimensions", n_freq, dk);
    SLLM_REQUIRE(layout == 0 || layout == 1, SLLM_EINVAL, "seq_normed_rotary_kv: layout 0 (interleaved) or 1 (halves)");
    SLLM_REQUIRE(kv_dtype == SLLM_F32 || kv_dtype == SLLM_BF16, SLLM_ENOTSUP, "seq_normed_rotary_kv: fp32 or bf16 pools");
    SLLM_REQUIRE(dk <= 8192, SLLM_ENOTSUP, "seq_normed_rotary_kv: heads of %d", dk);
    const dim3 grid(b->T, (heads + 2 * kv_heads + 3) / 4);
    const size_t smem = 4 * (size_t)dk * sizeof(float);
    if (kv_dtype == SLLM_F32)
        seq_normed_rotary_kv_kernel<float><<<grid, 128, smem, as_stream(stream)>>>(*b, q, ldq, heads, dk, k, ldk, kv_heads, v, ldv, dv, q_norm_w, k_norm_w, eps, freq,
                                                                                 n_freq, layout, (float*)k_pool, (float*)v_pool);
    else
        seq_normed_rotary_kv_kernel<uint16_t><<<grid, 128, smem, as_stream(stream)>>>(*b, q, ldq, heads, dk, k, ldk, kv_heads, v, ldv, dv, q_norm_w, k_norm_w, eps, freq,
                                                                                    n_freq, layout, (uint16_t*)k_pool, (uint16_t*)v_pool);
    ++g_launches;
    SLLM_LAUNCH_CHECK();
    return SLLM_OK;
}

int sllm_seq_angles(const sllm_seq_batch* b, const double* freq, int32_t n_freq, float* out, sllm_stream_t stream) {
    SLLM_REQUIRE(b && b->T > 0 && b->tok_pos && freq && out && n_freq > 0 && (uintptr_t)out % 8 == 0, SLLM_EINVAL, "seq_angles: bad argument");
    seq_angles_kernel<<<(b->T * n_freq + 127) / 128, 128, 0, as_stream(stream)>>>(*b, freq, n_freq, (float2*)out);
    ++g_launches;
    SLLM_LAUNCH_CHECK();
    return SLLM_OK;
}

int sllm_seq_wide_normed_rotary_kv(const sllm_seq_batch* b, float* q, int32_t ldq, int32_t heads, int32_t dk, const float* k, int32_t ldk, int32_t kv_heads,
                                   const float* v, int32_t ldv, int32_t dv, const float* q_norm_w, const float* k_norm_w, float eps, const float* angles,
                                   int32_t n_freq, int32_t layout, float* v_shared, int32_t share, float lambda, const float* talk, void* q_mixed,
                                   int32_t k_joint, void* k_pool, void* v_pool, int32_t kv_dtype, sllm_stream_t stream) {
    SLLM_REQUIRE(b && b->T > 0 && b->tok_slot && b->tok_pos && b->block_table, SLLM_EINVAL, "seq_wide_normed_rotary_kv: incomplete batch description");
    SLLM_REQUIRE(q && k && v && k_pool && v_pool && heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dk > 0 && dv > 0, SLLM_EINVAL,
                 "seq_wide_normed_rotary_kv: bad argument");
    SLLM_REQUIRE(n_freq >= 0 && 2 * n_freq <= dk && (n_freq == 0 || angles), SLLM_EINVAL, "seq_wide_normed_rotary_kv: %d rotary pairs do not fit %d dimensions", n_freq, dk);
    SLLM_REQUIRE(layout == 0 || layout == 1, SLLM_EINVAL, "seq_wide_normed_rotary_kv: layout 0 (interleaved) or 1 (halves)");
    SLLM_REQUIRE(share >= 0 && share <= 2 && (share == 0 || v_shared), SLLM_EINVAL, "seq_wide_normed_rotary_kv: share 0 (none), 1 (write) or 2 (blend) with a buffer");
    SLLM_REQUIRE(!q_mixed || (talk && (uintptr_t)q_mixed % 16 == 0), SLLM_EINVAL, "seq_wide_normed_rotary_kv: mixed queries need the mixing matrix and an aligned buffer");
    SLLM_REQUIRE(kv_dtype == SLLM_F32 || kv_dtype == SLLM_BF16, SLLM_ENOTSUP, "seq_wide_normed_rotary_kv: fp32 or bf16 pools");
    const size_t smem = ((((size_t)heads * dk + 3) & ~(size_t)3) + (q_mixed ? (size_t)heads * heads : 0)) * sizeof(float);
    SLLM_REQUIRE(smem <= (size_t)smem_optin_bytes() - 1024, SLLM_ENOTSUP, "seq_wide_normed_rotary_kv: %d heads of %d do not fit shared memory", heads, dk);
    auto aligned = [](const void* x) { return x == nullptr || ((uintptr_t)x % 16) == 0; };
    const int vec = dk % 4 == 0 && dv % 4 == 0 && ldq % 4 == 0 && ldk % 4 == 0 && ldv % 4 == 0 && aligned(q) && aligned(k) && aligned(v) && aligned(q_norm_w) &&
                    aligned(k_norm_w) && aligned(v_shared) && aligned(k_pool) && aligned(v_pool);
#define SLLM_WIDE_LAUNCH(KV)                                                                                                                               \
    do {                                                                                                                                                   \
        if (smem > 48 * 1024)                                                                                                                              \
            SLLM_CUDA(cudaFuncSetAttribute(seq_wide_normed_rotary_kv_kernel<KV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));                 \
        seq_wide_normed_rotary_kv_kernel<KV><<<dim3(b->T, 2), 256, smem, as_stream(stream)>>>(*b, q, ldq, heads, dk, k, ldk, kv_heads, v, ldv, dv, q_norm_w, \
                                                                                             k_norm_w, eps, (const float2*)angles, n_freq, layout, v_shared, share, lambda, talk, \
                                                                                             (uint16_t*)q_mixed, k_joint, (KV*)k_pool, (KV*)v_pool, vec);   \
    } while (0)
    if (kv_dtype == SLLM_F32) SLLM_WIDE_LAUNCH(float);
    else SLLM_WIDE_LAUNCH(uint16_t);
#undef SLLM_WIDE_LAUNCH
    ++g_launches;
    SLLM_LAUNCH_CHECK();
    return SLLM_OK;
}

int sllm_seq_conv_rotary_kv(const sllm_seq_batch* b, const float* q, int32_t ldq, int32_t heads, int32_t dk, const float* k, int32_t ldk, int32_t kv_heads,
                            const float* v, int32_t ldv, int32_t dv, const float* conv_w, int32_t taps, float* ring, const float* angles, int32_t n_freq,
                            int32_t layout, int32_t unit, float eps, float* q_out, int32_t ldqo, void* k_pool, void* v_pool, int32_t kv_dtype,
                            sllm_stream_t stream) {
    SLLM_REQUIRE(b && b->T > 0 && b->tok_slot && b->tok_pos && b->block_table, SLLM_EINVAL, "seq_conv_rotary_kv: incomplete batch description");
    SLLM_REQUIRE(q && k && v && q_out && k_pool && v_pool && heads > 0 && kv_heads > 0 && dk > 0 && dv > 0, SLLM_EINVAL, "seq_conv_rotary_kv: bad argument");
    SLLM_REQUIRE(n_freq >= 0 && 2 * n_freq <= dk && (n_freq == 0 || angles), SLLM_EINVAL, "seq_conv_rotary_kv: %d rotary pairs do not fit %d dimensions", n_freq, dk);
    SLLM_REQUIRE(layout == 0 || layout == 1, SLLM_EINVAL, "seq_conv_rotary_kv: layout 0 (interleaved) or 1 (halves)");
    SLLM_REQUIRE(!conv_w || (taps >= 1 && (taps == 1 || ring) && q_out != q), SLLM_EINVAL, "seq_conv_rotary_kv: a convolution needs its ring and an output of its own");
    SLLM_REQUIRE(kv_dtype == SLLM_F32 || kv_dtype == SLLM_BF16, SLLM_ENOTSUP, "seq_conv_rotary_kv: fp32 or bf16 pools");
    SLLM_REQUIRE(dk <= 2048 && dv <= 2048, SLLM_ENOTSUP, "seq_conv_rotary_kv: heads of %d / %d", dk, dv);
    auto aligned = [](const void* x) { return x == nullptr || ((uintptr_t)x % 16) == 0; };
    const int vec = dk % 4 == 0 && dv % 4 == 0 && ldq % 4 == 0 && ldk % 4 == 0 && ldv % 4 == 0 && ldqo % 4 == 0 && aligned(q) && aligned(k) && aligned(v) &&
                    aligned(conv_w) && aligned(ring) && aligned(q_out) && aligned(k_pool) && aligned(v_pool);
    const int tile = b->T >= 512 ? 8 : 1;
    ConvRotaryArgs p{*b, q, k, v, ldq, ldk, ldv, heads, kv_heads, dk, dv, conv_w, taps, conv_w && taps > 1 ? ring : nullptr, conv_w && taps > 1 && b->T == b->nseg,
                     (const float2*)angles, n_freq, layout, unit, eps, q_out, ldqo, k_pool, v_pool, tile, vec};
    const dim3 grid((b->T + tile - 1) / tile, (heads + 2 * kv_heads + 3) / 4);
    const size_t smem = 4 * (size_t)((std::max(dk, dv) + 3) & ~3) * sizeof(float);
    if (vec && layout == 0 && dk <= 128 && dv <= 128 && (!conv_w || taps <= 4)) {
#define SLLM_ROW_LAUNCH(TAPS)                                                                                               \
    do {                                                                                                                    \
        if (kv_dtype == SLLM_F32) seq_conv_rotary_kv_row_kernel<float, TAPS><<<grid, 128, 0, as_stream(stream)>>>(p);       \
        else seq_conv_rotary_kv_row_kernel<uint16_t, TAPS><<<grid, 128, 0, as_stream(stream)>>>(p);                         \
    } while (0)
        if (!conv_w) SLLM_ROW_LAUNCH(0);
        else if (taps == 1) SLLM_ROW_LAUNCH(1);
        else if (taps == 2) SLLM_ROW_LAUNCH(2);
        else if (taps == 3) SLLM_ROW_LAUNCH(3);
        else SLLM_ROW_LAUNCH(4);
#undef SLLM_ROW_LAUNCH
        ++g_launches;
        SLLM_LAUNCH_CHECK();
        return SLLM_OK;
    }
    if (kv_dtype == SLLM_F32) seq_conv_rotary_kv_kernel<float><<<grid, 128, smem, as_stream(stream)>>>(p);
    else seq_conv_rotary_kv_kernel<uint16_t><<<grid, 128, smem, as_stream(stream)>>>(p);
    ++g_launches;
    SLLM_LAUNCH_CHECK();
    return SLLM_OK;
}

int sllm_seq_head_mix(const float* in, int32_t ldi, const float* mix, int32_t heads, int32_t kv_heads, int32_t dv, float* out, int32_t ldo, void* out16,
                      int32_t T, sllm_stream_t stream) {
    SLLM_REQUIRE(in && mix && (out || out16) && T > 0 && heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dv > 0, SLLM_EINVAL, "seq_head_mix: bad argument");
    SLLM_REQUIRE(heads <= 96, SLLM_ENOTSUP, "seq_head_mix: %d heads beyond 96", heads);
    const int threads = T >= 64 ? 256 : std::min(1024, std::max(128, (heads * dv + 31) / 32 * 32));
    seq_head_mix_kernel<<<T, threads, (size_t)heads * heads * sizeof(float), as_stream(stream)>>>(in, ldi, mix, heads, kv_heads, dv, out, ldo, (uint16_t*)out16, T);
    ++g_launches;
    SLLM_LAUNCH_CHECK();
    return SLLM_OK;
}

}  // extern "C"
