// csrc/seq_chunk.cu — the delta rule (decay per head or per key channel) and linear attention with a constant decay, in blocks of 16 tokens
// on the tensor cores: portions of prompts in bf16 mode. Within a block that starts from the state S0 [dk][dv], with G_i the running sum of
// the logarithms of the decays (a vector over the key channels) up to token i,
//     u_i = beta_i (v_i - S0^T (e^G_i k_i) - sum_{j<i} A_ij u_j),       A_ij = sum_c k_ic k_jc e^(G_ic - G_jc)
//     o_i = S0^T (e^G_i q_i) + sum_{j<=i} B_ij u_j,                     B_ij = sum_c q_ic k_jc e^(G_ic - G_jc)
//     S'  = e^G_n S0 + sum_j (e^(G_n - G_j) k_j) u_j^T
// (e^G per key channel, i.e. on the rows of S). The u of a block solve a 16 x 16 triangular system, u = M (v - S0^T (e^G k)); linear attention
// is the case M = 1, no S0 term in u. No factor exceeds 1: a difference of sums is formed before its exponential.
//
// (1) seq_chunk_prepare_kernel, CTA = (block, head), all blocks of the step in parallel: silu / rotation / unit vectors, G, A and B (fp32,
// a pair of threads per entry), M by forward substitution; leaves e^G k, e^G q, e^(G_n - G) k, M and B as the tensor-core fragments the walk
// will load, each as two bf16 terms (x = hi + lo, |x - hi - lo| <= 2^-17 |x|), and e^G_n in fp32.
// (2) seq_chunk_walk_kernel, CTA = (portion, head, 64 value columns), warp = 16 value columns: S^T [16][dk] stays in the accumulators
// (fp32) from the portion's first token to its last. An accumulator fragment is register for register an A fragment of the next product, so
// state, u and o never leave the warp; all products take both operands as two bf16 terms (three products, fp32 accumulation), which keeps
// the recurrence at fp32 working accuracy. The blocks' records arrive by cp.async, three stages.
#include "seq_attn.cuh"
#include "seq_chunk.cuh"

namespace sllm {

constexpr int kPrepThreads = 288;    // two threads per entry of a triangle of 16 x 16
constexpr int kWalkStages = 3, kWalkCols = 64;
constexpr float kLog2e = 1.4426950408889634f;

struct ChunkPlace { int seg, start, n, id; };      // segment, first token in the batch, tokens, number of the block in segment order
__device__ __forceinline__ ChunkPlace chunk_place(const sllm_seq_batch& b, int item) {
    ChunkPlace c;
    const int tile = item >> 1, half = item & 1;
    c.seg = b.qt_seg[tile];
    const int off = b.qt_off[tile] + half * kChunk;
    c.n = min(kChunk, b.seg_len[c.seg] - off);
    c.start = b.seg_start[c.seg] + off;
    c.id = 2 * (b.seg_tile0[c.seg] + b.qt_off[tile] / 32) + half;
    return c;
}

// eight values -> 16 bytes of hi terms and 16 bytes of lo terms
__device__ __forceinline__ void chunk_put(uint8_t* hi, uint8_t* lo, int at, const float (&v)[8]) {
    uint32_t h[4], l[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) split_bf16(v[2 * i], v[2 * i + 1], &h[i], &l[i]);
    reinterpret_cast<uint4*>(hi)[at] = make_uint4(h[0], h[1], h[2], h[3]);
    reinterpret_cast<uint4*>(lo)[at] = make_uint4(l[0], l[1], l[2], l[3]);
}

template <bool kDelta>
__global__ void __launch_bounds__(kPrepThreads) seq_chunk_prepare_kernel(ChunkArgs p) {
    extern __shared__ __align__(16) float cp_sm[];
    __shared__ float s_A[kChunk][kChunk + 1], s_B[kChunk][kChunk + 1], s_M[kChunk][kChunk + 1], s_beta[kChunk];
    const sllm_seq_batch& b = p.b;
    const ChunkPlace c = chunk_place(b, blockIdx.x);
    if (c.n <= 0) return;
    const int h = blockIdx.y, kvh = h / (p.heads / p.kv_heads), dk = p.dk, dkp = chunk_key(dk), ld = dkp + 4;
    float* s_k = cp_sm;                 // [16][ld]
    float* s_q = s_k + kChunk * ld;     // [16][ld]
    float* s_G = s_q + kChunk * ld;     // [16][ld], delta rule only
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float rate = kDelta ? expf(p.A_log[h]) : p.rate[h];
    const float lg = -rate * kLog2e;    // constant decay: its base-2 logarithm
    for (int i = threadIdx.x; i < kChunk * dkp; i += kPrepThreads) {
        const int tok = i / dkp, ch = i % dkp;
        const bool has = tok < c.n && ch < dk;
        const size_t t = (size_t)(c.start + tok);
        float kv = has ? p.k[t * p.ldk + (size_t)kvh * dk + ch] : 0.0f, qv = has ? p.q[t * p.ldq + (size_t)kvh * dk + ch] : 0.0f;
        if (!kDelta && p.silu) {
            kv = kv * seq_sigmoid(kv);
            qv = qv * seq_sigmoid(qv);
        }
        s_k[tok * ld + ch] = kv;
        s_q[tok * ld + ch] = qv;
        if (kDelta) {
            float g = 0.0f;
            if (has) {
                const int at = p.channel ? h * dk + ch : h;
                g = lg * seq_softplus(p.al[t * p.lda + at] + p.dt_bias[at]);
            }
            s_G[tok * ld + ch] = g;
        }
    }
    if (kDelta && threadIdx.x < kChunk) s_beta[threadIdx.x] = (int)threadIdx.x < c.n ? seq_sigmoid(p.bl[(size_t)(c.start + threadIdx.x) * p.ldb + h]) : 0.0f;
    __syncthreads();
    for (int tok = warp; tok < c.n; tok += kPrepThreads / 32) {
        float* kr = s_k + tok * ld;
        float* qr = s_q + tok * ld;
        if (kDelta) {                                    // unit vectors
            float sk = 0.0f, sq = 0.0f;
            for (int ch = lane; ch < dk; ch += 32) {
                sk = fmaf(kr[ch], kr[ch], sk);
                sq = fmaf(qr[ch], qr[ch], sq);
            }
            const float ik = 1.0f / sqrtf(warp_sum(sk) + p.unit_eps), iq = p.scale / sqrtf(warp_sum(sq) + p.unit_eps);
            for (int ch = lane; ch < dk; ch += 32) {
                kr[ch] *= ik;
                qr[ch] *= iq;
            }
        } else {
            for (int i = lane; i < p.n_freq; i += 32) {
                const int ia = p.layout == 0 ? 2 * i : i, ib = p.layout == 0 ? 2 * i + 1 : i + p.n_freq;
                const float2 a = p.angles[(size_t)(c.start + tok) * p.n_freq + i];
                const float ku = kr[ia], kw = kr[ib], qu = qr[ia], qw = qr[ib];
                kr[ia] = ku * a.x - kw * a.y;
                kr[ib] = kw * a.x + ku * a.y;
                qr[ia] = qu * a.x - qw * a.y;
                qr[ib] = qw * a.x + qu * a.y;
            }
            __syncwarp();
            if (p.scale != 1.0f)
                for (int ch = lane; ch < dk; ch += 32) kr[ch] *= p.scale;
        }
    }
    if (kDelta && threadIdx.x >= kPrepThreads - 128 && (int)threadIdx.x - (kPrepThreads - 128) < dkp) {   // running sums (a column no other thread touches)
        float* col = s_G + threadIdx.x - (kPrepThreads - 128);
        float sum = 0.0f;
#pragma unroll
        for (int i = 0; i < kChunk; ++i) {
            sum += col[i * ld];
            col[i * ld] = sum;
        }
    }
    __syncthreads();
    // the two matrices: two threads per entry (i >= j), each half of the channels in groups of four
    {
        const int e = threadIdx.x >> 1, part = threadIdx.x & 1;
        int i = (int)((sqrtf(8.0f * e + 1.0f) - 1.0f) * 0.5f);
        while ((i + 1) * (i + 2) / 2 <= e) ++i;
        while (i * (i + 1) / 2 > e) --i;
        const int j = e - i * (i + 1) / 2;
        float a = 0.0f, bb = 0.0f;
        if (i < kChunk) {
            const float4 *ki = reinterpret_cast<const float4*>(s_k + i * ld), *kj = reinterpret_cast<const float4*>(s_k + j * ld), *qi = reinterpret_cast<const float4*>(s_q + i * ld);
            const float4 *Gi = reinterpret_cast<const float4*>(s_G + i * ld), *Gj = reinterpret_cast<const float4*>(s_G + j * ld);
            for (int g = part; g < dkp / 4; g += 2) {
                float4 x = kj[g];
                const float4 y = qi[g];
                if (kDelta) {
                    const float4 ga = Gi[g], gb = Gj[g], z = ki[g];
                    x = make_float4(x.x * exp2f(ga.x - gb.x), x.y * exp2f(ga.y - gb.y), x.z * exp2f(ga.z - gb.z), x.w * exp2f(ga.w - gb.w));
                    a = fmaf(z.x, x.x, fmaf(z.y, x.y, fmaf(z.z, x.z, fmaf(z.w, x.w, a))));
                }
                bb = fmaf(y.x, x.x, fmaf(y.y, x.y, fmaf(y.z, x.z, fmaf(y.w, x.w, bb))));
            }
        }
        a += __shfl_xor_sync(0xffffffffu, a, 1);
        bb += __shfl_xor_sync(0xffffffffu, bb, 1);
        if (i < kChunk && part == 0) {
            s_A[i][j] = a;
            s_B[i][j] = kDelta ? bb : bb * exp2f(lg * (float)(i - j));
            if (i != j) s_B[j][i] = 0.0f;
        }
    }
    __syncthreads();
    uint8_t* rec = p.ws + ((size_t)c.id * p.heads + h) * chunk_record_bytes(dkp);
    const size_t plane = (size_t)kChunk * dkp * 2;
    uint8_t* mats = rec + 6 * plane;                     // M hi, M lo, B hi, B lo: 512 bytes each
    float* D = reinterpret_cast<float*>(mats + 4 * kChunk * kChunk * 2);
    if (kDelta && warp == 0) {                           // M = (1 + diag(beta) A)^-1 diag(beta), lane = column
        float m[kChunk];
#pragma unroll
        for (int i = 0; i < kChunk; ++i) {
            float acc = 0.0f;
#pragma unroll
            for (int l = 0; l < i; ++l) acc = fmaf(s_A[i][l], m[l], acc);
            m[i] = s_beta[i] * ((i == lane ? 1.0f : 0.0f) - acc);
            if (lane < kChunk) s_M[i][lane] = m[i];
        }
    }
    const int last = c.n - 1;
    // logarithm of the decay from the block's start to after token i, and from after token i to the block's end
    auto G = [&](int i, int ch) { return kDelta ? s_G[i * ld + ch] : lg * (float)(min(i, last) + 1); };
    const int granules = dkp * 2;                        // 16-byte pieces of a plane: [k-step][lane]
    for (int x = threadIdx.x; x < 3 * granules; x += kPrepThreads) {
        const int which = x / granules, at = x % granules, ks = at >> 5, gr = (at & 31) >> 2, cc = at & 3;
        float v[8];
#pragma unroll
        for (int y = 0; y < 4; ++y) {                    // pairs: (first / second group of 8) x (first / second half of the k-step)
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int outer = (y >> 1) * 8 + gr, inner = (y & 1) * 8 + 2 * cc + half;
                if (which < 2) {
                    const int tok = outer, ch = ks * 16 + inner;
                    v[2 * y + half] = (which == 0 ? s_k : s_q)[tok * ld + ch] * exp2f(G(tok, ch));
                } else {
                    const int tok = inner, ch = ks * 16 + outer;
                    v[2 * y + half] = s_k[tok * ld + ch] * exp2f(G(last, ch) - G(tok, ch));
                }
            }
        }
        if (!kDelta && which == 0) continue;             // no S0 term in u
        chunk_put(rec + 2 * which * plane, rec + (2 * which + 1) * plane, at, v);
    }
    for (int ch = threadIdx.x; ch < dkp; ch += kPrepThreads) D[ch] = exp2f(G(last, ch));
    __syncthreads();
    for (int x = threadIdx.x; x < 64; x += kPrepThreads) {
        const int which = x >> 5, gr = (x & 31) >> 2, cc = x & 3;
        if (!kDelta && which == 0) continue;
        float v[8];
#pragma unroll
        for (int y = 0; y < 4; ++y)
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int i = (y >> 1) * 8 + gr, j = (y & 1) * 8 + 2 * cc + half;
                v[2 * y + half] = which == 0 ? s_M[i][j] : s_B[i][j];
            }
        chunk_put(mats + 2 * which * 512, mats + (2 * which + 1) * 512, x & 31, v);
    }
}

// three products of two-term operands: (ah + al) (bh + bl) without al * bl, each into an accumulator of its own (no product waits for another)
__device__ __forceinline__ void mma_split(float (&d)[4], float (&dl)[4], float (&dm)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], uint32_t h0, uint32_t h1, uint32_t l0, uint32_t l1) {
    mma_bf16_16816(d, ah, h0, h1);
    mma_bf16_16816(dl, al, h0, h1);
    mma_bf16_16816(dm, ah, l0, l1);
}

// KS: k-steps of 16 key channels
template <int KS, bool kDelta>
__global__ void __launch_bounds__(128) seq_chunk_walk_kernel(ChunkArgs p, int vec) {
    extern __shared__ __align__(16) uint8_t cw_sm[];
    constexpr int dkp = KS * 16;
    constexpr uint32_t kPlane = kChunk * dkp * 2;
    const size_t rec_bytes = chunk_record_bytes(dkp);
    const size_t stage_bytes = rec_bytes + kChunk * kWalkCols * 4;
    const sllm_seq_batch& b = p.b;
    const int seg = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * kWalkCols;
    const int start = b.seg_start[seg], len = b.seg_len[seg], slot = b.seg_slot[seg];
    const int blocks = (len + kChunk - 1) / kChunk;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, c = lane & 3;
    const int cl = warp * 16 + g, r0 = col0 + cl, r1 = r0 + 8;      // this thread's two value columns
    const bool ok0 = r0 < p.dv, ok1 = r1 < p.dv;
    const uint8_t* recs = p.ws + ((size_t)(2 * b.seg_tile0[seg]) * p.heads + h) * rec_bytes;
    auto issue = [&](int blk) {
        uint8_t* dst = cw_sm + (size_t)(blk % kWalkStages) * stage_bytes;
        const uint8_t* src = recs + (size_t)blk * p.heads * rec_bytes;
        for (uint32_t i = threadIdx.x + (kDelta ? 0 : 2 * kPlane / 16); i < rec_bytes / 16; i += 128) cp_async16(dst + 16 * i, src + 16 * i, 16);
        float* dv = reinterpret_cast<float*>(dst + rec_bytes);
        const int n = min(kChunk, len - blk * kChunk);
        if (vec) {
            for (int i = threadIdx.x; i < kChunk * kWalkCols / 4; i += 128) {
                const int tok = i / (kWalkCols / 4), j = (i % (kWalkCols / 4)) * 4;
                const bool has = tok < n && col0 + j < p.dv;
                cp_async16(dv + tok * kWalkCols + j, has ? p.v + (size_t)(start + blk * kChunk + tok) * p.ldv + (size_t)h * p.dv + col0 + j : p.v, has ? 16 : 0);
            }
        } else {
            for (int i = threadIdx.x; i < kChunk * kWalkCols; i += 128) {
                const int tok = i / kWalkCols, j = i % kWalkCols;
                const bool has = tok < n && col0 + j < p.dv;
                const float* s = has ? p.v + (size_t)(start + blk * kChunk + tok) * p.ldv + (size_t)h * p.dv + col0 + j : p.v;
                asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(smem_u32(dv + i)), "l"(s), "r"(has ? 4 : 0) : "memory");
            }
        }
        cp_async_commit();
    };
    issue(0);
    if (blocks > 1) issue(1);
    else cp_async_commit();
    float* st = p.state + ((size_t)slot * p.heads + h) * p.dk * p.dv;
    float S[2 * KS][4];                                  // S^T: rows r0 / r1, columns (key channels) nt * 8 + 2c, + 1
#pragma unroll
    for (int nt = 0; nt < 2 * KS; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int ch = nt * 8 + 2 * c + (e & 1);
            S[nt][e] = (e < 2 ? ok0 : ok1) && ch < p.dk ? st[(size_t)ch * p.dv + (e < 2 ? r0 : r1)] : 0.0f;
        }
    for (int blk = 0; blk < blocks; ++blk) {
        cp_async_wait<1>();
        __syncthreads();                                 // this block has landed for everyone, and everyone has left the block before
        if (blk + 2 < blocks) issue(blk + 2);
        else cp_async_commit();
        const uint8_t* rec = cw_sm + (size_t)(blk % kWalkStages) * stage_bytes;
        const uint4* Kh = reinterpret_cast<const uint4*>(rec) + lane;
        const uint4* Kl = Kh + kPlane / 16;
        const uint4* Qh = Kl + kPlane / 16;
        const uint4* Ql = Qh + kPlane / 16;
        const uint4* Eh = Ql + kPlane / 16;              // keys decayed to the block's end
        const uint4* El = Eh + kPlane / 16;
        const uint4* Mh = El + kPlane / 16;              // M hi, M lo, B hi, B lo: 32 pieces each
        const float* D = reinterpret_cast<const float*>(rec + 6 * kPlane + 4 * kChunk * kChunk * 2);
        const float* sv = reinterpret_cast<const float*>(rec + rec_bytes);
        const int n = min(kChunk, len - blk * kChunk);
        if (col0 + warp * 16 < p.dv) {                   // the same answer in every lane of the warp
        float x[2][4] = {}, xl[2][4] = {}, xm[2][4] = {}, o[2][4] = {}, ol[2][4] = {}, om[2][4] = {};     // rows r0 / r1, columns (tokens) nt * 8 + 2c, + 1
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
            uint32_t ah[4], al[4];
            split_bf16(S[2 * ks][0], S[2 * ks][1], &ah[0], &al[0]);
            split_bf16(S[2 * ks][2], S[2 * ks][3], &ah[1], &al[1]);
            split_bf16(S[2 * ks + 1][0], S[2 * ks + 1][1], &ah[2], &al[2]);
            split_bf16(S[2 * ks + 1][2], S[2 * ks + 1][3], &ah[3], &al[3]);
            if (kDelta) {
                const uint4 kh = Kh[ks * 32], kl = Kl[ks * 32];
                mma_split(x[0], xl[0], xm[0], ah, al, kh.x, kh.y, kl.x, kl.y);
                mma_split(x[1], xl[1], xm[1], ah, al, kh.z, kh.w, kl.z, kl.w);
            }
            const uint4 qh = Qh[ks * 32], ql = Ql[ks * 32];
            mma_split(o[0], ol[0], om[0], ah, al, qh.x, qh.y, ql.x, ql.y);
            mma_split(o[1], ol[1], om[1], ah, al, qh.z, qh.w, ql.z, ql.w);
        }
#pragma unroll
        for (int nt = 0; nt < 2 * KS; ++nt) {            // the old state decays to the block's end
            const float2 d = *reinterpret_cast<const float2*>(D + nt * 8 + 2 * c);
            S[nt][0] *= d.x;
            S[nt][1] *= d.y;
            S[nt][2] *= d.x;
            S[nt][3] *= d.y;
        }
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                float v = sv[(nt * 8 + 2 * c + (e & 1)) * kWalkCols + cl + (e < 2 ? 0 : 8)];
                if (!kDelta && p.silu) v = v * seq_sigmoid(v);
                x[nt][e] = v - (x[nt][e] + (xl[nt][e] + xm[nt][e]));
            }
        uint32_t uh[4], ul[4];
        auto operand = [&](const float (&y)[2][4]) {     // rows x 16 tokens as an A fragment
            split_bf16(y[0][0], y[0][1], &uh[0], &ul[0]);
            split_bf16(y[0][2], y[0][3], &uh[1], &ul[1]);
            split_bf16(y[1][0], y[1][1], &uh[2], &ul[2]);
            split_bf16(y[1][2], y[1][3], &uh[3], &ul[3]);
        };
        operand(x);
        if (kDelta) {
            float u[2][4] = {}, lo[2][4] = {}, mid[2][4] = {};
            const uint4 mh = Mh[0], ml = Mh[32];
            mma_split(u[0], lo[0], mid[0], uh, ul, mh.x, mh.y, ml.x, ml.y);
            mma_split(u[1], lo[1], mid[1], uh, ul, mh.z, mh.w, ml.z, ml.w);
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) u[nt][e] += lo[nt][e] + mid[nt][e];
            operand(u);
        }
        const uint4 bh = Mh[64], bl = Mh[96];
        mma_split(o[0], ol[0], om[0], uh, ul, bh.x, bh.y, bl.x, bl.y);
        mma_split(o[1], ol[1], om[1], uh, ul, bh.z, bh.w, bl.z, bl.w);
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
            const uint4 eh = Eh[ks * 32], el = El[ks * 32];
            mma_bf16_16816(S[2 * ks], uh, eh.x, eh.y);
            mma_bf16_16816(S[2 * ks + 1], uh, eh.z, eh.w);
            mma_bf16_16816(S[2 * ks], ul, eh.x, eh.y);
            mma_bf16_16816(S[2 * ks + 1], ul, eh.z, eh.w);
            mma_bf16_16816(S[2 * ks], uh, el.x, el.y);
            mma_bf16_16816(S[2 * ks + 1], uh, el.z, el.w);
        }
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int tok = nt * 8 + 2 * c + (e & 1);
                if (tok < n && (e < 2 ? ok0 : ok1)) p.o[(size_t)(start + blk * kChunk + tok) * p.ldo + (size_t)h * p.dv + (e < 2 ? r0 : r1)] = o[nt][e] + (ol[nt][e] + om[nt][e]);
            }
        }
    }
#pragma unroll
    for (int nt = 0; nt < 2 * KS; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int ch = nt * 8 + 2 * c + (e & 1);
            if ((e < 2 ? ok0 : ok1) && ch < p.dk) st[(size_t)ch * p.dv + (e < 2 ? r0 : r1)] = S[nt][e];
        }
}

int launch_chunk_scan(const ChunkArgs& p, cudaStream_t st) {
    const int dkp = chunk_key(p.dk);
    SLLM_REQUIRE(p.dk <= kChunkMaxKey && p.ws && ((uintptr_t)p.ws % 16) == 0 && p.b.seg_tile0 && p.b.qt_seg && p.b.qt_off && p.b.n_qtiles > 0, SLLM_EINVAL,
                 "chunk scan: heads of %d key channels, or an incomplete batch description", p.dk);
    const size_t smem_prep = (size_t)3 * kChunk * (dkp + 4) * sizeof(float);
    const size_t smem_walk = kWalkStages * (chunk_record_bytes(dkp) + kChunk * kWalkCols * 4);
    const dim3 gp(2 * p.b.n_qtiles, p.heads), gw(p.b.nseg, p.heads, (p.dv + kWalkCols - 1) / kWalkCols);
    if (p.delta) seq_chunk_prepare_kernel<true><<<gp, kPrepThreads, smem_prep, st>>>(p);
    else seq_chunk_prepare_kernel<false><<<gp, kPrepThreads, smem_prep, st>>>(p);
    ++g_launches;
    SLLM_LAUNCH_CHECK();
    const int vec = p.ldv % 4 == 0 && p.dv % 4 == 0 && ((uintptr_t)p.v % 16) == 0;
#define SLLM_CHUNK_LAUNCH(KS, DELTA)                                                                                                                      \
    do {                                                                                                                                                  \
        SLLM_CUDA(cudaFuncSetAttribute(seq_chunk_walk_kernel<KS, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_walk));                   \
        seq_chunk_walk_kernel<KS, DELTA><<<gw, 128, smem_walk, st>>>(p, vec);                                                                             \
    } while (0)
#define SLLM_CHUNK_LAUNCH_KS(DELTA)                          \
    do {                                                     \
        if (dkp == 32) SLLM_CHUNK_LAUNCH(2, DELTA);          \
        else if (dkp == 64) SLLM_CHUNK_LAUNCH(4, DELTA);     \
        else if (dkp == 96) SLLM_CHUNK_LAUNCH(6, DELTA);     \
        else SLLM_CHUNK_LAUNCH(8, DELTA);                    \
    } while (0)
    if (p.delta) SLLM_CHUNK_LAUNCH_KS(true);
    else SLLM_CHUNK_LAUNCH_KS(false);
#undef SLLM_CHUNK_LAUNCH_KS
#undef SLLM_CHUNK_LAUNCH
    ++g_launches;
    SLLM_LAUNCH_CHECK();
    return SLLM_OK;
}

}  // namespace sllm

extern "C" int64_t sllm_seq_chunk_ws_bytes(int32_t n_qtiles, int32_t heads, int32_t dk) {
    return dk > 0 && dk <= sllm::kChunkMaxKey && n_qtiles > 0 && heads > 0 ? (int64_t)sllm::chunk_ws_bytes(n_qtiles, heads, dk) : 0;
}
