// csrc/seq_sublayer.cu — the seam between two sublayers of a model whose sublayers are wrapped in scalar RMS norms and read their input
// through a short causal convolution: x <- x + g_post * y / rms(y) (the residual sum, fp32), then h = n + conv(n) with
// n = g_pre * x / rms(x) and conv a per-channel causal convolution over time, as ONE kernel. A norm here has one number as its weight.
// The same seam serves pre-norm layers: the sum may take y as it is (no norm on the sublayer's output), and the norm in front of the
// next sublayer may carry a weight per channel stored as its distance from a constant, n = g_pre * (offset + w[c]) * x / rms(x); and layers
// whose only norm sits on the sublayer's OUTPUT, with a weight per channel: x <- x + g_post * w[c] * y / rms(y), the next sublayer reading x
// itself (the seam then leaves x as bf16 operand rows). Layers whose sublayers run side by side on one norm's output have a seam of their
// own (sllm_seq_branch_seam): the sum of several branches, each normed or not, with a weight per channel, then the next layer's norm.
//
// The convolution reaches taps-1 tokens back. Inside a portion those are rows of this step: a CTA (one per token) recomputes the
// residual sum and the norm of its predecessors from the sublayer's input and output (x is therefore read from one buffer and written to
// another). Before the portion they come from the sequence's state: a ring of taps-1 normed rows per slot, position p at row
// p % (taps-1). A ring may not be written while other CTAs of the launch still read it, so the normed rows of a portion's last tokens
// go to a per-token stash, and the NEXT seam launch moves them into the ring (`flush_*`); the model's last seam (the final norm, no
// convolution) flushes the last ring.
#include "seq_common.cuh"

namespace sllm {

struct SeamArgs {
    sllm_seq_batch b;
    const float* x_in; float* x_out;          // residual stream before / after the sum (x_out unused when y is NULL)
    const float* y; float post_g;             // sublayer output and its norm's weight; NULL = no sum
    int has_pre; float pre_g, eps;            // 0 = only the sum
    const float* conv_w; int taps;            // [d][taps], last column = the current token; NULL = no convolution
    const float* ring;                        // [slots][taps-1][d]
    float* h; uint16_t* h16;                  // what the next sublayer reads, fp32 and (optionally) as bf16 operand rows
    float* stash;                             // [T][d]: normed rows of tokens that a later launch moves into `ring`
    float* flush_ring; int flush_taps;        // the ring that takes the stash the previous seam left
    int d;
    int post_norm;                            // 0 = y is added as it is
    const float* pre_w; float pre_off;        // [d] or NULL: channel c of the normed row is also multiplied by pre_off + pre_w[c]
    const float* post_w;                      // [d] or NULL: channel c of the normed sublayer output is also multiplied by post_w[c]
};

__device__ __forceinline__ float seam_gain(const SeamArgs& p, int j) { return p.pre_w ? p.pre_off + p.pre_w[j] : 1.0f; }

__device__ __forceinline__ float seam_post(const SeamArgs& p, int j) { return p.post_w ? p.post_w[j] : 1.0f; }

// is token t among the last `keep` tokens of its portion?
__device__ __forceinline__ bool seam_is_last(const sllm_seq_batch& b, int t, int slot, int keep) {
    return keep > 0 && (t + keep >= b.T || b.tok_slot[t + keep] != slot);
}

__global__ void seq_seam_kernel(SeamArgs p) {
    extern __shared__ __align__(16) float seam_sm[];   // [d] the row at hand, [d] the convolution's sums
    __shared__ float red[33];
    float* s_row = seam_sm;
    float* s_acc = seam_sm + p.d;
    const sllm_seq_batch& b = p.b;
    const int t = blockIdx.x, d = p.d, slot = b.tok_slot[t], pos = b.tok_pos[t];
    // the stash of the previous seam goes into that seam's ring before this launch overwrites the stash row
    if (p.flush_ring && seam_is_last(b, t, slot, p.flush_taps - 1)) {
        float* dst = p.flush_ring + ((size_t)slot * (p.flush_taps - 1) + pos % (p.flush_taps - 1)) * d;
        for (int j = threadIdx.x; j < d; j += blockDim.x) dst[j] = p.stash[(size_t)t * d + j];
    }
    const int reach = (p.has_pre && p.conv_w) ? p.taps - 1 : 0;
    bool started = false;                                // does s_acc hold a sum yet? (the same answer in every thread)
    for (int back = reach; back >= 0; --back) {          // the current token last: its normed row stays in s_row
        if (pos - back < 0) continue;                    // before the sequence's start: zeros
        const bool here = back == 0 || (t - back >= 0 && b.tok_slot[t - back] == slot);
        if (!here) {
            const float* src = p.ring + ((size_t)slot * (p.taps - 1) + (pos - back) % (p.taps - 1)) * d;
            for (int j = threadIdx.x; j < d; j += blockDim.x) {
                s_acc[j] = fmaf(p.conv_w[(size_t)j * p.taps + p.taps - 1 - back], src[j], started ? s_acc[j] : 0.0f);
            }
            started = true;
            continue;
        }
        const size_t r = (size_t)(t - back) * d;
        float inv_y = 1.0f;
        if (p.y && p.post_norm) {
            float ss = 0.0f;
            for (int j = threadIdx.x; j < d; j += blockDim.x) ss = fmaf(p.y[r + j], p.y[r + j], ss);
            inv_y = p.post_g / sqrtf(block_sum(ss, red) / (float)d + p.eps);
        }
        float ss = 0.0f;
        for (int j = threadIdx.x; j < d; j += blockDim.x) {
            float v = p.x_in[r + j];
            if (p.y) {
                v = fmaf(p.y[r + j] * seam_post(p, j), inv_y, v);
                if (back == 0) p.x_out[r + j] = v;
            }
            if (!p.has_pre && p.h16) p.h16[r + j] = f32_to_bf16_bits(v);
            s_row[j] = v;
            ss = fmaf(v, v, ss);
        }
        if (!p.has_pre) return;
        const float inv = p.pre_g / sqrtf(block_sum(ss, red) / (float)d + p.eps);
        if (!p.conv_w) {
            for (int j = threadIdx.x; j < d; j += blockDim.x) {
                const float v = s_row[j] * inv * seam_gain(p, j);
                p.h[r + j] = v;
                if (p.h16) p.h16[r + j] = f32_to_bf16_bits(v);
            }
            return;
        }
        const bool keep = back == 0 && seam_is_last(b, t, slot, p.taps - 1);
        for (int j = threadIdx.x; j < d; j += blockDim.x) {
            const float n = s_row[j] * inv * seam_gain(p, j);
            float acc = fmaf(p.conv_w[(size_t)j * p.taps + p.taps - 1 - back], n, started ? s_acc[j] : 0.0f);
            if (back == 0) {
                acc += n;
                p.h[r + j] = acc;
                if (p.h16) p.h16[r + j] = f32_to_bf16_bits(acc);
                if (keep) p.stash[r + j] = n;
            } else {
                s_acc[j] = acc;
            }
        }
        started = true;
    }
}

// ---- the same seam without a convolution or a ring, rows of a multiple of four floats: the row stays in registers ----------------------------
// CTA = token, R groups of four channels per thread; x and y are read once, in flight together, and everything is stored once.
template <int R>
__global__ void __launch_bounds__(1024) seq_seam_row_kernel(SeamArgs p) {
    __shared__ float red[33];
    const int d4 = p.d / 4;
    const size_t r = (size_t)blockIdx.x * p.d;
    float x[R][4], y[R][4];
    float sy = 0.0f;
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int j = threadIdx.x + i * blockDim.x;
        const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        const float4 xv = j < d4 ? *reinterpret_cast<const float4*>(p.x_in + r + 4 * j) : zero;
        const float4 yv = j < d4 && p.y ? *reinterpret_cast<const float4*>(p.y + r + 4 * j) : zero;
        x[i][0] = xv.x; x[i][1] = xv.y; x[i][2] = xv.z; x[i][3] = xv.w;
        y[i][0] = yv.x; y[i][1] = yv.y; y[i][2] = yv.z; y[i][3] = yv.w;
#pragma unroll
        for (int e = 0; e < 4; ++e) sy = fmaf(y[i][e], y[i][e], sy);
    }
    auto pack = [&](const float (&v)[4]) {
        return make_uint2((uint32_t)f32_to_bf16_bits(v[0]) | ((uint32_t)f32_to_bf16_bits(v[1]) << 16), (uint32_t)f32_to_bf16_bits(v[2]) | ((uint32_t)f32_to_bf16_bits(v[3]) << 16));
    };
    float ss = 0.0f;
    if (p.y) {
        const float inv_y = p.post_norm ? p.post_g / sqrtf(block_sum(sy, red) / (float)p.d + p.eps) : 1.0f;
#pragma unroll
        for (int i = 0; i < R; ++i) {
            const int j = threadIdx.x + i * blockDim.x;
            if (j >= d4) continue;
            const float4 w = p.post_w ? *reinterpret_cast<const float4*>(p.post_w + 4 * j) : make_float4(1.0f, 1.0f, 1.0f, 1.0f);
            x[i][0] = fmaf(y[i][0] * w.x, inv_y, x[i][0]);
            x[i][1] = fmaf(y[i][1] * w.y, inv_y, x[i][1]);
            x[i][2] = fmaf(y[i][2] * w.z, inv_y, x[i][2]);
            x[i][3] = fmaf(y[i][3] * w.w, inv_y, x[i][3]);
            *reinterpret_cast<float4*>(p.x_out + r + 4 * j) = make_float4(x[i][0], x[i][1], x[i][2], x[i][3]);
        }
    }
    if (!p.has_pre) {
        if (p.h16)
#pragma unroll
            for (int i = 0; i < R; ++i) {
                const int j = threadIdx.x + i * blockDim.x;
                if (j < d4) *reinterpret_cast<uint2*>(p.h16 + r + 4 * j) = pack(x[i]);
            }
        return;
    }
#pragma unroll
    for (int i = 0; i < R; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) ss = fmaf(x[i][e], x[i][e], ss);     // channels beyond the row are zeros
    const float inv = p.pre_g / sqrtf(block_sum(ss, red) / (float)p.d + p.eps);
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int j = threadIdx.x + i * blockDim.x;
        if (j >= d4) continue;
        const float4 w = p.pre_w ? *reinterpret_cast<const float4*>(p.pre_w + 4 * j) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        const float off = p.pre_w ? p.pre_off : 1.0f;
        const float v[4] = {x[i][0] * inv * (off + w.x), x[i][1] * inv * (off + w.y), x[i][2] * inv * (off + w.z), x[i][3] * inv * (off + w.w)};
        *reinterpret_cast<float4*>(p.h + r + 4 * j) = make_float4(v[0], v[1], v[2], v[3]);
        if (p.h16) *reinterpret_cast<uint2*>(p.h16 + r + 4 * j) = pack(v);
    }
}

// ---- the same seam as two launches, for steps of many tokens: no row is normed more than once ------------------------------------------
// (1) one CTA per token: the residual sum and the scale of the next norm, scale[t] = g_pre / rms(x_new[t]);
// (2) element-wise over (token, channel): h = n + conv(n) with n = scale * x_new read from the step's rows (complete after launch 1) or
//     the ring, the stash and the flush as in the one-launch form.
__global__ void seq_seam_sum_kernel(SeamArgs p, float* __restrict__ scale) {
    extern __shared__ __align__(16) float seam_sm[];   // [d] the sublayer's output row
    __shared__ float red[33];
    const int t = blockIdx.x, d = p.d;
    const size_t r = (size_t)t * d;
    float ss = 0.0f;
    if (p.y) {
        float sy = 0.0f;
        for (int j = threadIdx.x; j < d; j += blockDim.x) {
            const float v = p.y[r + j];
            seam_sm[j] = v;
            sy = fmaf(v, v, sy);
        }
        const float inv_y = p.post_norm ? p.post_g / sqrtf(block_sum(sy, red) / (float)d + p.eps) : 1.0f;
        for (int j = threadIdx.x; j < d; j += blockDim.x) {
            const float v = fmaf(seam_sm[j] * seam_post(p, j), inv_y, p.x_in[r + j]);
            p.x_out[r + j] = v;
            ss = fmaf(v, v, ss);
        }
    } else {
        for (int j = threadIdx.x; j < d; j += blockDim.x) ss = fmaf(p.x_in[r + j], p.x_in[r + j], ss);
    }
    ss = block_sum(ss, red);
    if (threadIdx.x == 0) scale[t] = p.pre_g / sqrtf(ss / (float)d + p.eps);
}

constexpr int kSeamMaxTaps = 64;

// The rows a token's convolution reads are found once per CTA (the step's own rows with their scales, or ring rows), then the channels
// are walked four at a time with 16-byte loads where the row length allows.
__global__ void seq_seam_conv_kernel(SeamArgs p, const float* __restrict__ scale, int vec) {
    __shared__ const float* s_src[kSeamMaxTaps];   // [back] row that lies `back` positions before the token, NULL = before the sequence's start
    __shared__ float s_mul[kSeamMaxTaps];
    __shared__ bool back_is_step[kSeamMaxTaps];    // the row is one of this step's (not yet normed) rather than a ring row
    const sllm_seq_batch& b = p.b;
    const int t = blockIdx.x, d = p.d, slot = b.tok_slot[t], pos = b.tok_pos[t], taps = p.taps;
    const float* x = p.y ? p.x_out : p.x_in;             // the stream after the sum
    const bool flush = p.flush_ring && seam_is_last(b, t, slot, p.flush_taps - 1);
    const bool keep = seam_is_last(b, t, slot, taps - 1);
    float* fdst = flush ? p.flush_ring + ((size_t)slot * (p.flush_taps - 1) + pos % (p.flush_taps - 1)) * d : nullptr;
    const size_t r = (size_t)t * d;
    if ((int)threadIdx.x < taps) {
        const int back = threadIdx.x;
        const float* src = nullptr;
        float mul = 1.0f;
        bool in_step = false;
        if (pos - back >= 0) {
            if (back == 0 || (t - back >= 0 && b.tok_slot[t - back] == slot)) {
                src = x + r - (size_t)back * d;
                mul = scale[t - back];
                in_step = true;
            } else {
                src = p.ring + ((size_t)slot * (taps - 1) + (pos - back) % (taps - 1)) * d;
            }
        }
        s_src[back] = src;
        s_mul[back] = mul;
        back_is_step[back] = in_step;
    }
    __syncthreads();
    const float own = s_mul[0];
    if (vec) {
        for (int j = (blockIdx.y * blockDim.x + threadIdx.x) * 4; j < d; j += gridDim.y * blockDim.x * 4) {
            if (flush) *reinterpret_cast<float4*>(fdst + j) = *reinterpret_cast<const float4*>(p.stash + r + j);
            float acc[4] = {0.0f, 0.0f, 0.0f, 0.0f};
            const float gn[4] = {seam_gain(p, j), seam_gain(p, j + 1), seam_gain(p, j + 2), seam_gain(p, j + 3)};
            for (int back = taps - 1; back >= 1; --back) {
                const float* src = s_src[back];
                if (!src) continue;
                const float4 v = *reinterpret_cast<const float4*>(src + j);
                const float m = s_mul[back];
                // a ring row is normed and weighted already (its multiplier is 1); a row of this step gets the channel's weight here
                const bool raw = back_is_step[back];
                const float n4[4] = {v.x * m * (raw ? gn[0] : 1.0f), v.y * m * (raw ? gn[1] : 1.0f), v.z * m * (raw ? gn[2] : 1.0f), v.w * m * (raw ? gn[3] : 1.0f)};
#pragma unroll
                for (int e = 0; e < 4; ++e) acc[e] = fmaf(p.conv_w[(size_t)(j + e) * taps + taps - 1 - back], n4[e], acc[e]);
            }
            const float4 v = *reinterpret_cast<const float4*>(x + r + j);
            const float n4[4] = {v.x * own * gn[0], v.y * own * gn[1], v.z * own * gn[2], v.w * own * gn[3]};
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[e] = fmaf(p.conv_w[(size_t)(j + e) * taps + taps - 1], n4[e], acc[e]) + n4[e];
            *reinterpret_cast<float4*>(p.h + r + j) = make_float4(acc[0], acc[1], acc[2], acc[3]);
            if (p.h16) {
                const uint2 packed = make_uint2((uint32_t)f32_to_bf16_bits(acc[0]) | ((uint32_t)f32_to_bf16_bits(acc[1]) << 16),
                                                (uint32_t)f32_to_bf16_bits(acc[2]) | ((uint32_t)f32_to_bf16_bits(acc[3]) << 16));
                *reinterpret_cast<uint2*>(p.h16 + r + j) = packed;
            }
            if (keep) *reinterpret_cast<float4*>(p.stash + r + j) = make_float4(n4[0], n4[1], n4[2], n4[3]);
        }
        return;
    }
    for (int j = blockIdx.y * blockDim.x + threadIdx.x; j < d; j += gridDim.y * blockDim.x) {
        if (flush) fdst[j] = p.stash[r + j];
        float acc = 0.0f;
        const float gn = seam_gain(p, j);
        for (int back = taps - 1; back >= 1; --back) {
            const float* src = s_src[back];
            if (src) acc = fmaf(p.conv_w[(size_t)j * taps + taps - 1 - back], src[j] * s_mul[back] * (back_is_step[back] ? gn : 1.0f), acc);
        }
        const float n = x[r + j] * own * gn;
        acc = fmaf(p.conv_w[(size_t)j * taps + taps - 1], n, acc) + n;
        p.h[r + j] = acc;
        if (p.h16) p.h16[r + j] = f32_to_bf16_bits(acc);
        if (keep) p.stash[r + j] = n;
    }
}


// ---- the seam of a layer whose sublayers run side by side -------------------------------------------------------------------------------
// x <- x + sum_i gain_i * (branch i, or branch i / rms(branch i)), gain_i a weight per channel (a layer scale, a constant factor and a norm's
// weight are one product), then h = w * x / rms(x) for the next layer, fp32 and / or as bf16 operand rows. CTA = token; the row and its
// branches stay in registers, E channels at a time, R groups per thread; the branches' root mean squares are ONE reduction.
constexpr int kMaxBranches = 4;
struct BranchSeamArgs {
    const float* x_in; float* x_out;                 // may be the same rows: a CTA owns its row
    int n; const float* y[kMaxBranches]; const float* gain[kMaxBranches]; int normed[kMaxBranches];
    float eps;
    const float* norm_w; float* h; uint16_t* h16;    // norm_w NULL = only the sum
    int d;
};

template <int E, int R>
__global__ void __launch_bounds__(E * R <= 8 ? 1024 : 512) seq_branch_seam_kernel(BranchSeamArgs p) {
    __shared__ float s_part[kMaxBranches][33];
    __shared__ float red[33];
    const int groups = p.d / E, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = blockDim.x >> 5;
    const size_t r = (size_t)blockIdx.x * p.d;
    auto load = [&](const float* src, int j, float (&v)[E]) {
        if (E == 4) {
            const float4 f = *reinterpret_cast<const float4*>(src + 4 * j);
            v[0] = f.x; v[1 % E] = f.y; v[2 % E] = f.z; v[3 % E] = f.w;
        } else {
            v[0] = src[j];
        }
    };
    float x[R][E], y[kMaxBranches][R][E];
    float ss[kMaxBranches];
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int j = threadIdx.x + i * blockDim.x;
#pragma unroll
        for (int e = 0; e < E; ++e) x[i][e] = 0.0f;
        if (j < groups) load(p.x_in + r, j, x[i]);
    }
#pragma unroll
    for (int k = 0; k < kMaxBranches; ++k) {
        ss[k] = 0.0f;
#pragma unroll
        for (int i = 0; i < R; ++i) {
            const int j = threadIdx.x + i * blockDim.x;
#pragma unroll
            for (int e = 0; e < E; ++e) y[k][i][e] = 0.0f;
            if (k < p.n && j < groups) load(p.y[k] + r, j, y[k][i]);
#pragma unroll
            for (int e = 0; e < E; ++e) ss[k] = fmaf(y[k][i][e], y[k][i][e], ss[k]);
        }
    }
    bool any = false;
    for (int k = 0; k < p.n; ++k) any |= p.normed[k] != 0;
    if (any) {                                           // the same answer in every thread
#pragma unroll
        for (int k = 0; k < kMaxBranches; ++k) {
            const float v = warp_sum(ss[k]);
            if (lane == 0) s_part[k][warp] = v;
        }
        __syncthreads();
        if (warp < kMaxBranches) {
            const float v = warp_sum(lane < nwarps ? s_part[warp][lane] : 0.0f);
            if (lane == 0) s_part[warp][32] = v;
        }
        __syncthreads();
    }
#pragma unroll
    for (int k = 0; k < kMaxBranches; ++k) {
        if (k >= p.n) continue;
        const float inv = p.normed[k] ? 1.0f / sqrtf(s_part[k][32] / (float)p.d + p.eps) : 1.0f;
#pragma unroll
        for (int i = 0; i < R; ++i) {
            const int j = threadIdx.x + i * blockDim.x;
            if (j >= groups) continue;
            float g[E];
            load(p.gain[k], j, g);
#pragma unroll
            for (int e = 0; e < E; ++e) x[i][e] = fmaf(y[k][i][e] * inv, g[e], x[i][e]);
        }
    }
    float sx = 0.0f;
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int j = threadIdx.x + i * blockDim.x;
#pragma unroll
        for (int e = 0; e < E; ++e) sx = fmaf(x[i][e], x[i][e], sx);     // channels beyond the row are zeros
        if (j >= groups) continue;
        if (E == 4) *reinterpret_cast<float4*>(p.x_out + r + 4 * j) = make_float4(x[i][0], x[i][1 % E], x[i][2 % E], x[i][3 % E]);
        else p.x_out[r + j] = x[i][0];
    }
    if (!p.norm_w) return;
    const float inv = 1.0f / sqrtf(block_sum(sx, red) / (float)p.d + p.eps);
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int j = threadIdx.x + i * blockDim.x;
        if (j >= groups) continue;
        float w[E];
        load(p.norm_w, j, w);
#pragma unroll
        for (int e = 0; e < E; ++e) w[e] = (x[i][e] * inv) * w[e];
        if (E == 4) {
            if (p.h) *reinterpret_cast<float4*>(p.h + r + 4 * j) = make_float4(w[0], w[1 % E], w[2 % E], w[3 % E]);
            if (p.h16) *reinterpret_cast<uint2*>(p.h16 + r + 4 * j) = make_uint2(pack_bf16(w[0], w[1 % E]), pack_bf16(w[2 % E], w[3 % E]));
        } else {
            if (p.h) p.h[r + j] = w[0];
            if (p.h16) p.h16[r + j] = f32_to_bf16_bits(w[0]);
        }
    }
}

}  // namespace sllm

using namespace sllm;

extern "C" int sllm_seq_branch_seam(const float* x_in, float* x_out, int32_t n, const float* const* y, const float* const* gain, const int32_t* normed, float eps,
                                    const float* norm_w, float* h, void* h16, int32_t T, int32_t d, sllm_stream_t stream) {
    SLLM_REQUIRE(x_in && x_out && T > 0 && d > 0 && n >= 0 && (n == 0 || (y && gain && normed)), SLLM_EINVAL, "seq_branch_seam: bad argument");
    SLLM_REQUIRE(n <= kMaxBranches, SLLM_ENOTSUP, "seq_branch_seam: %d branches beyond %d", n, kMaxBranches);
    SLLM_REQUIRE(!norm_w || h || h16, SLLM_EINVAL, "seq_branch_seam: no output for the normed rows");
    SLLM_REQUIRE(d <= 16384, SLLM_ENOTSUP, "seq_branch_seam: rows of %d floats beyond 16384", d);
    BranchSeamArgs p{};
    auto aligned = [](const void* q) { return q == nullptr || ((uintptr_t)q % 16) == 0; };
    bool vec = d % 4 == 0 && aligned(x_in) && aligned(x_out) && aligned(norm_w) && aligned(h) && aligned(h16);
    for (int i = 0; i < n; ++i) {
        SLLM_REQUIRE(y[i] && gain[i], SLLM_EINVAL, "seq_branch_seam: branch %d is missing", i);
        p.y[i] = y[i]; p.gain[i] = gain[i]; p.normed[i] = normed[i];
        vec = vec && aligned(y[i]) && aligned(gain[i]);
    }
    p.x_in = x_in; p.x_out = x_out; p.n = n; p.eps = eps; p.norm_w = norm_w; p.h = h; p.h16 = (uint16_t*)h16; p.d = d;
    // many tokens: CTAs of 256 threads with up to four groups of channels each; few: a thread per group of channels (at least a warp per branch)
    const int items = vec ? d / 4 : d;
    int cta = T >= 64 ? std::max(std::min(items, 256), (items + 3) / 4) : items;
    cta = std::min(items > 2048 ? 512 : 1024, std::max(128, (cta + 31) / 32 * 32));
    const int per = (items + cta - 1) / cta;
    SLLM_REQUIRE(per <= (vec ? 8 : 32), SLLM_ENOTSUP, "seq_branch_seam: rows of %d floats", d);
    cudaStream_t st = as_stream(stream);
#define SLLM_BRANCH_LAUNCH(E, R) seq_branch_seam_kernel<E, R><<<T, cta, 0, st>>>(p)
    if (vec) {
        if (per == 1) SLLM_BRANCH_LAUNCH(4, 1);
        else if (per == 2) SLLM_BRANCH_LAUNCH(4, 2);
        else if (per <= 4) SLLM_BRANCH_LAUNCH(4, 4);
        else SLLM_BRANCH_LAUNCH(4, 8);
    } else {
        if (per <= 4) SLLM_BRANCH_LAUNCH(1, 4);
        else SLLM_BRANCH_LAUNCH(1, 32);
    }
#undef SLLM_BRANCH_LAUNCH
    ++g_launches;
    SLLM_LAUNCH_CHECK();
    return SLLM_OK;
}

extern "C" int sllm_seq_seam(const sllm_seq_batch* b, const float* x_in, float* x_out, const float* y, float post_g, int32_t has_pre, float pre_g,
                             float eps, const float* conv_w, int32_t taps, const float* ring, float* h, void* h16, float* stash, float* flush_ring,
                             int32_t flush_taps, int32_t d, float* scales, int32_t post_norm, const float* pre_w, float pre_w_offset, const float* post_w,
                             sllm_stream_t stream) {
    SLLM_REQUIRE(b && b->T > 0 && b->tok_slot && b->tok_pos, SLLM_EINVAL, "seq_seam: incomplete batch description");
    SLLM_REQUIRE(x_in && d > 0 && (!y || (x_out && x_out != x_in)), SLLM_EINVAL, "seq_seam: the residual sum needs a second buffer for x");
    SLLM_REQUIRE(!has_pre || h, SLLM_EINVAL, "seq_seam: no output for the normed rows");
    SLLM_REQUIRE(!conv_w || (taps >= 1 && taps <= kSeamMaxTaps && (taps == 1 || (ring && stash))), SLLM_EINVAL, "seq_seam: a convolution (1..%d taps) needs its ring and a stash", kSeamMaxTaps);
    SLLM_REQUIRE(!flush_ring || (flush_taps >= 2 && stash), SLLM_EINVAL, "seq_seam: nothing to flush from");
    if (conv_w && taps == 1) ring = nullptr;
    const size_t smem = 2 * (size_t)d * sizeof(float);
    SLLM_REQUIRE(smem <= (size_t)smem_optin_bytes() - 1024, SLLM_ENOTSUP, "seq_seam: rows of %d floats do not fit shared memory", d);
    if (smem > 48 * 1024) SLLM_CUDA(cudaFuncSetAttribute(seq_seam_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    SeamArgs p{*b, x_in, x_out, y, post_g, has_pre, pre_g, eps, conv_w, taps, ring, h, (uint16_t*)h16, stash, flush_ring, flush_taps, d, post_norm, pre_w, pre_w_offset, post_w};
    auto aligned = [](const void* q) { return q == nullptr || ((uintptr_t)q % 16) == 0; };
    if (!conv_w && !flush_ring && d % 4 == 0 && d <= 4 * 4 * 1024 && aligned(x_in) && aligned(x_out) && aligned(y) && aligned(h) && aligned(h16) && aligned(pre_w) &&
        aligned(post_w)) {
        // many tokens: CTAs of 256 threads with up to four groups of channels each; few: a thread per group of channels
        const int d4 = d / 4, cta = std::min(1024, (((b->T >= 64 ? std::max(std::min(d4, 256), (d4 + 3) / 4) : d4) + 31) / 32) * 32), per = (d4 + cta - 1) / cta;
        if (per == 1) seq_seam_row_kernel<1><<<b->T, cta, 0, as_stream(stream)>>>(p);
        else if (per == 2) seq_seam_row_kernel<2><<<b->T, cta, 0, as_stream(stream)>>>(p);
        else seq_seam_row_kernel<4><<<b->T, cta, 0, as_stream(stream)>>>(p);
        ++g_launches;
        SLLM_LAUNCH_CHECK();
        return SLLM_OK;
    }
    const int threads = b->T >= 64 ? (d >= 2048 ? 256 : 128) : std::min(1024, std::max(128, (d + 31) / 32 * 32));
    if (scales && has_pre && conv_w && b->T >= 64 && b->T <= 65535) {       // many tokens: two launches, every row normed once
        seq_seam_sum_kernel<<<b->T, threads, smem / 2, as_stream(stream)>>>(p, scales);
        const int vec = d % 4 == 0 && aligned(x_in) && aligned(x_out) && aligned(ring) && aligned(h) && aligned(stash) && aligned(flush_ring) &&
                        (h16 == nullptr || ((uintptr_t)h16 % 8) == 0);
        seq_seam_conv_kernel<<<dim3(b->T, std::max(1, std::min(4, d / 4096))), 256, 0, as_stream(stream)>>>(p, scales, vec);
        g_launches += 2;
        SLLM_LAUNCH_CHECK();
        return SLLM_OK;
    }
    seq_seam_kernel<<<b->T, threads, smem, as_stream(stream)>>>(p);
    ++g_launches;
    SLLM_LAUNCH_CHECK();
    return SLLM_OK;
}
