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
// (2) seq_chunk_walk_kernel, CTA = (portion, head, 16 or 32 value columns), two or four warps = 16 value columns, a share of the key channels each: their part of
// S^T [16][dk] stays in the accumulators (fp32) from the portion's first token to its last. An accumulator fragment is register for register
// an A fragment of the next product, so state and u never leave the registers; all products take both operands as two bf16 terms (three products, fp32 accumulation), which keeps
// the recurrence at fp32 working accuracy. The blocks' records arrive by cp.async, three stages.
#include "seq_attn.cuh"
#include "seq_chunk.cuh"

namespace sllm {

constexpr int kPrepThreads = 288;    // two threads per entry of a triangle of 16 x 16
constexpr int kWalkStages = 3;
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

// vec: rows of q, k, v (and of the channels' steps) may be read 16 bytes at a time
template <bool kDelta, int dkp>
__global__ void __launch_bounds__(kPrepThreads) seq_chunk_prepare_kernel(ChunkArgs p, int vec) {
    extern __shared__ __align__(16) float cp_sm[];
    __shared__ float s_A[kChunk][kChunk + 1], s_B[kChunk][kChunk + 1], s_M[kChunk][kChunk + 1], s_beta[kChunk];
    const sllm_seq_batch& b = p.b;
    const ChunkPlace c = chunk_place(b, blockIdx.x);
    if (c.n <= 0) return;
    const int h = blockIdx.y, kvh = h / (p.heads / p.kv_heads), dk = p.dk;
    constexpr int ld = dkp + 4;
    float* s_k = cp_sm;                 // [16][ld]
    float* s_q = s_k + kChunk * ld;     // [16][ld]
    float* s_G = s_q + kChunk * ld;     // [16][ld], delta rule only
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float rate = kDelta ? expf(p.A_log[h]) : p.rate[h];
    const float lg = -rate * kLog2e;    // constant decay: its base-2 logarithm
    auto load4 = [&](const float* row, int ch, bool has) {             // channels ch .. ch + 3 of a row, zeros beyond the head
        float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (!has) return v;
        if (vec && ch < dk) return *reinterpret_cast<const float4*>(row + ch);
        if (ch < dk) v.x = row[ch];
        if (ch + 1 < dk) v.y = row[ch + 1];
        if (ch + 2 < dk) v.z = row[ch + 2];
        if (ch + 3 < dk) v.w = row[ch + 3];
        return v;
    };
    auto silu4 = [](float4 v) { return make_float4(v.x * seq_sigmoid(v.x), v.y * seq_sigmoid(v.y), v.z * seq_sigmoid(v.z), v.w * seq_sigmoid(v.w)); };
    for (int i = threadIdx.x; i < kChunk * dkp / 4; i += kPrepThreads) {
        const int tok = i / (dkp / 4), ch = (i % (dkp / 4)) * 4;
        const bool has = tok < c.n;
        const size_t t = (size_t)(c.start + (has ? tok : 0));
        float4 kv = load4(p.k + t * p.ldk + (size_t)kvh * dk, ch, has), qv = load4(p.q + t * p.ldq + (size_t)kvh * dk, ch, has);
        if (!kDelta && p.silu) {
            kv = silu4(kv);
            qv = silu4(qv);
        }
        *reinterpret_cast<float4*>(s_k + tok * ld + ch) = kv;
        *reinterpret_cast<float4*>(s_q + tok * ld + ch) = qv;
        if (kDelta) {
            float4 g = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (has && p.channel) {
                const float4 a = load4(p.al + t * p.lda + (size_t)h * dk, ch, true), bias = load4(p.dt_bias + (size_t)h * dk, ch, true);
                g = make_float4(ch < dk ? lg * seq_softplus(a.x + bias.x) : 0.0f, ch + 1 < dk ? lg * seq_softplus(a.y + bias.y) : 0.0f,
                                ch + 2 < dk ? lg * seq_softplus(a.z + bias.z) : 0.0f, ch + 3 < dk ? lg * seq_softplus(a.w + bias.w) : 0.0f);
            } else if (has) {
                g.x = g.y = g.z = g.w = lg * seq_softplus(p.al[t * p.lda + h] + p.dt_bias[h]);
            }
            *reinterpret_cast<float4*>(s_G + tok * ld + ch) = g;
        }
    }
    if (!kDelta && p.silu)                               // the values too, for the walk
        for (int tok = warp; tok < c.n; tok += kPrepThreads / 32) {
            const float* src = p.v + (size_t)(c.start + tok) * p.ldv + (size_t)h * p.dv;
            float* dst = p.v_ws + ((size_t)c.id * kChunk + tok) * p.heads * p.dv + (size_t)h * p.dv;
            if (vec)
                for (int j = 4 * lane; j < p.dv; j += 128) *reinterpret_cast<float4*>(dst + j) = silu4(*reinterpret_cast<const float4*>(src + j));
            else
                for (int j = lane; j < p.dv; j += 32) dst[j] = src[j] * seq_sigmoid(src[j]);
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
    constexpr int granules = dkp * 2;                    // 16-byte pieces of a plane: [k-step][lane]
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

// KS: k-steps of 16 key channels. PARTS warps share 16 value columns, each owning KS / PARTS of the k-steps; they add their parts of the
// products with the old state through shared memory and finish 16 / PARTS outputs per column each. GROUPS: how many times 16 columns a CTA takes.
template <int KS, int PARTS, int GROUPS, bool kDelta>
__global__ void __launch_bounds__(PARTS * GROUPS * 32) seq_chunk_walk_kernel(ChunkArgs p, int vec) {
    extern __shared__ __align__(16) uint8_t cw_sm[];
    constexpr int dkp = KS * 16, HS = KS / PARTS, kThreads = PARTS * GROUPS * 32, kCols = GROUPS * 16;
    constexpr uint32_t kPlane = kChunk * dkp * 2;
    constexpr uint32_t rec_bytes = (uint32_t)chunk_record_bytes(dkp), stage_bytes = rec_bytes + kChunk * kCols * 4;
    const sllm_seq_batch& b = p.b;
    const int seg = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * kCols;
    const int start = b.seg_start[seg], len = b.seg_len[seg], slot = b.seg_slot[seg];
    const int blocks = (len + kChunk - 1) / kChunk;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, c = lane & 3;
    const int group = warp % GROUPS, part = warp / GROUPS, k0 = part * HS;   // this warp's value columns and first k-step
    const int cl = group * 16 + g, r0 = col0 + cl, r1 = r0 + 8;              // this thread's two value columns
    const bool ok0 = r0 < p.dv, ok1 = r1 < p.dv;
    // what the warps of a group hand each other: [group][part][x, x, o, o][lane]
    float4* exchange = reinterpret_cast<float4*>(cw_sm + kWalkStages * stage_bytes) + group * (PARTS * 4 * 32) + lane;
    const size_t first = 2 * (size_t)b.seg_tile0[seg];   // number of the portion's first block
    const uint8_t* recs = p.ws + (first * p.heads + h) * rec_bytes;
    // values: the batch's rows, or those the preparation left (passed through silu), 16 rows per block
    const bool own_v = !kDelta && p.silu;
    const float* vsrc = own_v ? p.v_ws + first * kChunk * p.heads * p.dv + (size_t)h * p.dv + col0 : p.v + (size_t)start * p.ldv + (size_t)h * p.dv + col0;
    const size_t ldv = own_v ? (size_t)p.heads * p.dv : (size_t)p.ldv;
    auto issue = [&](int blk) {
        uint8_t* dst = cw_sm + (blk % kWalkStages) * stage_bytes;
        const uint8_t* src = recs + (size_t)blk * p.heads * rec_bytes;
#pragma unroll 4
        for (uint32_t i = threadIdx.x + (kDelta ? 0 : 2 * kPlane / 16); i < rec_bytes / 16; i += kThreads) cp_async16(dst + 16 * i, src + 16 * i, 16);
        float* dv = reinterpret_cast<float*>(dst + rec_bytes);
        const int n = min(kChunk, len - blk * kChunk);
        const float* vb = vsrc + (size_t)blk * kChunk * ldv;
        if (vec) {
            for (int i = threadIdx.x; i < kChunk * kCols / 4; i += kThreads) {
                const int tok = i / (kCols / 4), j = (i % (kCols / 4)) * 4;
                const bool has = tok < n && col0 + j < p.dv;
                cp_async16(dv + tok * kCols + j, has ? vb + tok * ldv + j : vsrc, has ? 16 : 0);
            }
        } else {
            for (int i = threadIdx.x; i < kChunk * kCols; i += kThreads) {
                const int tok = i / kCols, j = i % kCols;
                const bool has = tok < n && col0 + j < p.dv;
                asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(smem_u32(dv + i)), "l"(has ? vb + tok * ldv + j : p.v), "r"(has ? 4 : 0) : "memory");
            }
        }
        cp_async_commit();
    };
    issue(0);
    if (blocks > 1) issue(1);
    else cp_async_commit();
    float* st = p.state + ((size_t)slot * p.heads + h) * p.dk * p.dv;
    float S[2 * HS][4];                                  // S^T: rows r0 / r1, columns (key channels) k0 * 16 + nt * 8 + 2c, + 1
#pragma unroll
    for (int nt = 0; nt < 2 * HS; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int ch = k0 * 16 + nt * 8 + 2 * c + (e & 1);
            S[nt][e] = (e < 2 ? ok0 : ok1) && ch < p.dk ? st[(size_t)ch * p.dv + (e < 2 ? r0 : r1)] : 0.0f;
        }
    const bool work = col0 + group * 16 < p.dv;          // the same answer in all warps of a group
    // the outputs this warp finishes: tokens mt * 8 + 2c and + 1 of columns r0 and r1 (two parts) or of one of them (four)
    const int mt = PARTS == 4 ? part >> 1 : part, mrow = PARTS == 4 ? part & 1 : 0;
    float* orow = p.o + (size_t)(start + mt * 8 + 2 * c) * p.ldo + (size_t)h * p.dv + (mrow ? r1 : r0);
    for (int blk = 0; blk < blocks; ++blk, orow += (size_t)kChunk * p.ldo) {
        cp_async_wait<1>();
        __syncthreads();                                 // this block has landed for everyone, and everyone has left the block before
        if (blk + 2 < blocks) issue(blk + 2);
        else cp_async_commit();
        if (!work) continue;
        const uint8_t* rec = cw_sm + (blk % kWalkStages) * stage_bytes;
        const uint4* Kh = reinterpret_cast<const uint4*>(rec) + k0 * 32 + lane;
        const uint4* Kl = Kh + kPlane / 16;
        const uint4* Qh = Kl + kPlane / 16;
        const uint4* Ql = Qh + kPlane / 16;
        const uint4* Eh = Ql + kPlane / 16;              // keys decayed to the block's end
        const uint4* El = Eh + kPlane / 16;
        const uint4* Mh = reinterpret_cast<const uint4*>(rec + 6 * kPlane) + lane;              // M hi, M lo, B hi, B lo: 32 pieces each
        const float* D = reinterpret_cast<const float*>(rec + 6 * kPlane + 4 * kChunk * kChunk * 2) + k0 * 16 + 2 * c;
        const float* sv = reinterpret_cast<const float*>(rec + rec_bytes) + 2 * c * kCols + cl;
        float x[2][4] = {}, xl[2][4] = {}, xm[2][4] = {}, o[2][4] = {}, ol[2][4] = {}, om[2][4] = {};     // rows r0 / r1, columns (tokens) nt * 8 + 2c, + 1
#pragma unroll
        for (int ks = 0; ks < HS; ++ks) {
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
        auto sum3 = [](const float (&p0)[4], const float (&p1)[4], const float (&p2)[4]) {
            return make_float4(p0[0] + (p1[0] + p2[0]), p0[1] + (p1[1] + p2[1]), p0[2] + (p1[2] + p2[2]), p0[3] + (p1[3] + p2[3]));
        };
        float4* mine = exchange + part * 4 * 32;
        if (kDelta) {
            mine[0] = sum3(x[0], xl[0], xm[0]);
            mine[32] = sum3(x[1], xl[1], xm[1]);
        }
        mine[64] = sum3(o[0], ol[0], om[0]);
        mine[96] = sum3(o[1], ol[1], om[1]);
#pragma unroll
        for (int nt = 0; nt < 2 * HS; ++nt) {            // the old state decays to the block's end
            const float2 d = *reinterpret_cast<const float2*>(D + nt * 8);
            S[nt][0] *= d.x;
            S[nt][1] *= d.y;
            S[nt][2] *= d.x;
            S[nt][3] *= d.y;
        }
        float v[2][4];
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) v[nt][e] = sv[(nt * 8 + (e & 1)) * kCols + (e < 2 ? 0 : 8)];
        asm volatile("bar.sync %0, %1;" ::"r"(1 + group), "n"(PARTS * 32) : "memory");   // the warps of the group
        if (kDelta) {
#pragma unroll
            for (int nt = 0; nt < 2; ++nt) {
                float4 y = exchange[nt * 32];
#pragma unroll
                for (int q = 1; q < PARTS; ++q) {
                    const float4 z = exchange[(q * 4 + nt) * 32];
                    y = make_float4(y.x + z.x, y.y + z.y, y.z + z.z, y.w + z.w);
                }
                v[nt][0] -= y.x;
                v[nt][1] -= y.y;
                v[nt][2] -= y.z;
                v[nt][3] -= y.w;
            }
        }
        uint32_t uh[4], ul[4];
        auto operand = [&](const float (&y)[2][4]) {     // rows x 16 tokens as an A fragment
            split_bf16(y[0][0], y[0][1], &uh[0], &ul[0]);
            split_bf16(y[0][2], y[0][3], &uh[1], &ul[1]);
            split_bf16(y[1][0], y[1][1], &uh[2], &ul[2]);
            split_bf16(y[1][2], y[1][3], &uh[3], &ul[3]);
        };
        operand(v);
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
#pragma unroll
        for (int ks = 0; ks < HS; ++ks) {
            const uint4 eh = Eh[ks * 32], el = El[ks * 32];
            mma_bf16_16816(S[2 * ks], uh, eh.x, eh.y);
            mma_bf16_16816(S[2 * ks + 1], uh, eh.z, eh.w);
            mma_bf16_16816(S[2 * ks], ul, eh.x, eh.y);
            mma_bf16_16816(S[2 * ks + 1], ul, eh.z, eh.w);
            mma_bf16_16816(S[2 * ks], uh, el.x, el.y);
            mma_bf16_16816(S[2 * ks + 1], uh, el.z, el.w);
        }
        const uint4 bh = Mh[64], bl = Mh[96];
        float y[4] = {}, yl[4] = {}, ym[4] = {};
        if (mt == 0) mma_split(y, yl, ym, uh, ul, bh.x, bh.y, bl.x, bl.y);
        else mma_split(y, yl, ym, uh, ul, bh.z, bh.w, bl.z, bl.w);
        const int n = min(kChunk, len - blk * kChunk), tok = mt * 8 + 2 * c;
        if (PARTS == 4) {                                // two tokens of one column
            const float* at = reinterpret_cast<const float*>(exchange + (2 + mt) * 32) + 2 * mrow;
            float2 z = *reinterpret_cast<const float2*>(at);
#pragma unroll
            for (int q = 1; q < PARTS; ++q) {
                const float2 w = *reinterpret_cast<const float2*>(at + q * 4 * 32 * 4);
                z = make_float2(z.x + w.x, z.y + w.y);
            }
            const float o0 = (mrow ? y[2] + (yl[2] + ym[2]) : y[0] + (yl[0] + ym[0])) + z.x, o1 = (mrow ? y[3] + (yl[3] + ym[3]) : y[1] + (yl[1] + ym[1])) + z.y;
            if (mrow ? ok1 : ok0) {
                if (tok < n) orow[0] = o0;
                if (tok + 1 < n) orow[p.ldo] = o1;
            }
        } else {                                         // two tokens of both columns
            const float4 z0 = exchange[(2 + mt) * 32], z1 = exchange[(4 + 2 + mt) * 32];
            if (ok0 && tok < n) orow[0] = y[0] + (yl[0] + ym[0]) + (z0.x + z1.x);
            if (ok0 && tok + 1 < n) orow[p.ldo] = y[1] + (yl[1] + ym[1]) + (z0.y + z1.y);
            if (ok1 && tok < n) orow[8] = y[2] + (yl[2] + ym[2]) + (z0.z + z1.z);
            if (ok1 && tok + 1 < n) orow[p.ldo + 8] = y[3] + (yl[3] + ym[3]) + (z0.w + z1.w);
        }
    }
#pragma unroll
    for (int nt = 0; nt < 2 * HS; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int ch = k0 * 16 + nt * 8 + 2 * c + (e & 1);
            if ((e < 2 ? ok0 : ok1) && ch < p.dk) st[(size_t)ch * p.dv + (e < 2 ? r0 : r1)] = S[nt][e];
        }
}

template <int KS, int PARTS, int GROUPS, bool kDelta>
static int launch_walk(const ChunkArgs& p, int vec, cudaStream_t st) {
    constexpr size_t smem = kWalkStages * (chunk_record_bytes(KS * 16) + kChunk * GROUPS * 16 * 4) + GROUPS * PARTS * 4 * 32 * sizeof(float4);
    SLLM_CUDA(cudaFuncSetAttribute(seq_chunk_walk_kernel<KS, PARTS, GROUPS, kDelta>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    seq_chunk_walk_kernel<KS, PARTS, GROUPS, kDelta><<<dim3(p.b.nseg, p.heads, (p.dv + GROUPS * 16 - 1) / (GROUPS * 16)), PARTS * GROUPS * 32, smem, st>>>(p, vec);
    ++g_launches;
    SLLM_LAUNCH_CHECK();
    return SLLM_OK;
}

template <bool kDelta>
static int launch_chunk_as(ChunkArgs p, cudaStream_t st) {
    const int dkp = chunk_key(p.dk);
    p.v_ws = reinterpret_cast<float*>(p.ws + 2 * (size_t)p.b.n_qtiles * p.heads * chunk_record_bytes(dkp));
    auto aligned = [](const void* q) { return ((uintptr_t)q % 16) == 0; };
    const int vec_prep = p.dk % 4 == 0 && p.dv % 4 == 0 && p.ldq % 4 == 0 && p.ldk % 4 == 0 && p.ldv % 4 == 0 && aligned(p.q) && aligned(p.k) && aligned(p.v) &&
                         (!p.channel || (p.lda % 4 == 0 && aligned(p.al) && aligned(p.dt_bias)));
    const dim3 grid(2 * p.b.n_qtiles, p.heads);
    const size_t smem = (size_t)3 * kChunk * (dkp + 4) * sizeof(float);
    if (dkp == 32) seq_chunk_prepare_kernel<kDelta, 32><<<grid, kPrepThreads, smem, st>>>(p, vec_prep);
    else if (dkp == 64) seq_chunk_prepare_kernel<kDelta, 64><<<grid, kPrepThreads, smem, st>>>(p, vec_prep);
    else if (dkp == 96) seq_chunk_prepare_kernel<kDelta, 96><<<grid, kPrepThreads, smem, st>>>(p, vec_prep);
    else seq_chunk_prepare_kernel<kDelta, 128><<<grid, kPrepThreads, smem, st>>>(p, vec_prep);
    ++g_launches;
    SLLM_LAUNCH_CHECK();
    const bool own_v = !kDelta && p.silu;
    const int vec = p.dv % 4 == 0 && (own_v || (p.ldv % 4 == 0 && ((uintptr_t)p.v % 16) == 0));
    // a walk is a chain of dependent blocks: few heads are spread over the machine 16 value columns a CTA, many take 32 (every CTA of a head
    // loads all of the head's records)
    const bool narrow = (long long)p.b.nseg * p.heads * ((p.dv + 31) / 32) < sm_count() / 2;
    if (dkp == 32) return narrow ? launch_walk<2, 2, 1, kDelta>(p, vec, st) : launch_walk<2, 2, 2, kDelta>(p, vec, st);
    if (dkp == 64) return narrow ? launch_walk<4, 4, 1, kDelta>(p, vec, st) : launch_walk<4, 4, 2, kDelta>(p, vec, st);
    if (dkp == 96) return narrow ? launch_walk<6, 2, 1, kDelta>(p, vec, st) : launch_walk<6, 2, 2, kDelta>(p, vec, st);
    return narrow ? launch_walk<8, 4, 1, kDelta>(p, vec, st) : launch_walk<8, 4, 2, kDelta>(p, vec, st);
}

int launch_chunk_scan(const ChunkArgs& p, cudaStream_t st) {
    SLLM_REQUIRE(p.dk <= kChunkMaxKey && p.ws && ((uintptr_t)p.ws % 16) == 0 && p.b.seg_tile0 && p.b.qt_seg && p.b.qt_off && p.b.n_qtiles > 0, SLLM_EINVAL,
                 "chunk scan: heads of %d key channels, or an incomplete batch description", p.dk);
    return p.delta ? launch_chunk_as<true>(p, st) : launch_chunk_as<false>(p, st);
}

}  // namespace sllm

extern "C" int64_t sllm_seq_chunk_ws_bytes(int32_t n_qtiles, int32_t heads, int32_t dk, int32_t dv) {
    return dk > 0 && dk <= sllm::kChunkMaxKey && dv > 0 && n_qtiles > 0 && heads > 0 ? (int64_t)sllm::chunk_ws_bytes(n_qtiles, heads, dk, dv) : 0;
}
