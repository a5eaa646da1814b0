// csrc/seq_attn_talk.cu — softmax attention of the ragged token batch whose scores are mixed over the heads BEFORE the softmax:
// own_g(i, j) = scale * q_g(i) . k_u(j) for every query head g (u = its key head), score_h = sum_g talk[h][g] own_g, softmax over the keys
// the query sees (its window, or its chunk of positions), one more term exp(sink_h) in the denominator, head h's weights on the values of
// its own value head, the result times a sigmoid gate per column. Scores, mixing, weights and sums are fp32 whatever the cache holds.
// The keys of all heads of a token lie side by side in one pool row of kv_heads * dk elements.
//
// seq_attention_talk_mma_kernel (bf16 pools, steps that hold a portion of a prompt): the sum over the heads of a key head moves into the
// query, score_h = scale * sum_u (sum_{g of u} talk[h][g] q_g) . k_u, so that head h is ONE product of its mixed query (kv_heads * dk long,
// made by the preparation kernel) with the token's whole key row: a plain tensor-core product, nothing to exchange between heads, and every
// head reads the same key tile. CTA = (tile of 32 queries, 1, 2 or 4 heads of one value head, share of the key tiles), a warp per head
// holding 32 queries x 64 keys of scores and 32 x dv of output; query and key rows arrive in pieces of 64 columns through a three-stage
// cp.async ring (128-byte rows, 16-byte units swizzled by the row), the values of a tile with its first piece. The weights enter the
// second product as two bf16 terms (fp32 working accuracy). With one share the kernel normalises, gates and stores the result itself.
//
// seq_attention_talk_kernel (any size, fp32 or bf16; single tokens): CTA = (1, 2 or 4 queries, ALL heads, share of the key tiles). A tile of
// 32 keys of as many key heads as fit is staged by cp.async; a warp computes the scores of up to four query heads of a key head (a lane
// owns a key), leaves them in shared memory, the mix reads all heads' scores of a key back, and the online softmax runs there; the
// weighted sums accumulate in shared memory. Every key and value is read once per CTA whatever the number of heads.
#include "seq_attn.cuh"

namespace sllm {

extern int g_tune_seq_attn_mma;   // runtime.cu

struct TalkArgs {
    sllm_seq_batch b;
    const float* q; int ldq;
    const uint16_t* qm;       // mixed queries [T][heads][kv_heads * dk] (tensor-core form)
    int heads, kv_heads, dk, dv; float scale;
    const float* talk;        // [heads][heads]
    const void *k_pool, *v_pool;
    int nsplit; float* ws;
    int window, keep_first, chunk;
    // the merge, when the kernel finishes by itself
    const float* sink; const float* gate; int ldg; float* out; int ldo; uint16_t* out16;
    // geometry of the any-size form: queries per CTA, key / value heads staged at once, padded row lengths, does the mix matrix sit in shared memory
    int nq, gs, dkq, ldk, ldv, talk_in_smem;
};

// ---- tensor-core form ---------------------------------------------------------------------------------------------------------------------
constexpr int kTalkStages = 3, kTalkCols = 64;   // ring of pieces; columns per piece (128 bytes)

__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}

// 2^x; tiny results become zero
__device__ __forceinline__ float fast_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

constexpr int kTalkKeys = 64;   // keys per tile

template <int kDvTiles, int kHeads>   // dv <= 8 * kDvTiles (multiple of 8); kHeads heads (= warps) per CTA
__global__ void __launch_bounds__(32 * kHeads) seq_attention_talk_mma_kernel(TalkArgs p) {
    constexpr int kKeys = kTalkKeys, kThreads = 32 * kHeads, qrows = kHeads * kBQ;
    extern __shared__ __align__(128) uint16_t smh[];
    const sllm_seq_batch& b = p.b;
    const int qt = blockIdx.x, split = blockIdx.z;
    const int seg = b.qt_seg[qt], off = b.qt_off[qt];
    const int nq = min(kBQ, b.seg_len[seg] - off), t0 = b.seg_start[seg] + off, pos0 = b.seg_pos0[seg] + off, slot = b.seg_slot[seg];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, c = lane & 3;
    const int h0 = blockIdx.y * kHeads, h = h0 + warp, gv = h0 / (p.heads / p.kv_heads);
    const int dv = p.dv, dvt = dv / 8, ldv = dv + 8, wide = p.kv_heads * p.dk, pieces = (wide + kTalkCols - 1) / kTalkCols;
    constexpr int stage_elems = (qrows + kKeys) * kTalkCols;
    const int v_elems = kKeys * ldv, v_bufs = pieces == 1 ? 3 : 2;
    uint16_t* smv = smh + kTalkStages * stage_elems;
    const uint16_t* kp = reinterpret_cast<const uint16_t*>(p.k_pool);
    const uint16_t* vp = reinterpret_cast<const uint16_t*>(p.v_pool);
    const int last_pos = pos0 + nq - 1;
    const TileList tiles(pos0, last_pos, seq_row_window(pos0, p.window, p.chunk), p.keep_first, kKeys);
    const int my_tiles = tiles.n > split ? (tiles.n - split + p.nsplit - 1) / p.nsplit : 0, total = my_tiles * pieces;

    // piece `ip` of this CTA's tile number `it` -> stage `st`, asynchronously; rows that do not exist and columns beyond the row are zeros.
    // A thread copies the same 16-byte unit of a piece's rows in every pass over them, kRowStep rows apart.
    constexpr int kRowStep = kThreads / 8;
    const int my_row = threadIdx.x >> 3, my_unit = threadIdx.x & 7;
    auto issue = [&](int it, int ip, int st) {
        const int j0 = tiles.tile_of(split + it * p.nsplit) * kKeys, col = ip * kTalkCols + my_unit * 8;
        const bool col_ok = col < wide;
        uint16_t* sQ = smh + st * stage_elems;
        uint16_t* sK = sQ + qrows * kTalkCols;
        const uint16_t* qsrc = p.qm + ((size_t)t0 * p.heads + h0) * wide + col;
#pragma unroll
        for (int k = 0; k < qrows / kRowStep; ++k) {
            const int row = my_row + k * kRowStep, r = row & (kBQ - 1), hh = row / kBQ;
            const bool take = col_ok && r < nq;
            cp_async16(sQ + row * kTalkCols + ((my_unit ^ (row & 7)) << 3), take ? qsrc + (r * p.heads + hh) * wide : p.qm, take ? 16 : 0);
        }
        size_t krow[2], vrow[2];      // pages hold a multiple of 32 positions: one look-up per 32 keys
#pragma unroll
        for (int q = 0; q < 2; ++q) {
            const int j = j0 + 32 * q;
            const int page = j <= last_pos ? b.block_table[(size_t)slot * b.max_pages + j / b.page_len] : 0, in_page = j % b.page_len;
            krow[q] = ((size_t)page * b.page_len + in_page) * wide;
            vrow[q] = seq_pool_row(page, p.kv_heads, gv, b.page_len, in_page, dv);
        }
#pragma unroll
        for (int k = 0; k < kKeys / kRowStep; ++k) {
            const int row = my_row + k * kRowStep;
            const bool take = col_ok && j0 + row <= last_pos;
            cp_async16(sK + row * kTalkCols + ((my_unit ^ (row & 7)) << 3), take ? kp + (k * kRowStep >= 32 ? krow[1] : krow[0]) + (row & 31) * wide + col : kp, take ? 16 : 0);
        }
        if (ip == 0) {
            uint16_t* sV = smv + (it % v_bufs) * v_elems;
            for (int i = threadIdx.x; i < kKeys * dvt; i += kThreads) {
                const int row = i / dvt, cc = (i % dvt) * 8;
                const bool take = j0 + row <= last_pos;
                cp_async16(sV + row * ldv + cc, take ? vp + (row < 32 ? vrow[0] : vrow[1]) + (row & 31) * dv + cc : vp, take ? 16 : 0);
            }
        }
    };
    int nxt_tile = 0, nxt_piece = 0, nxt_stage = 0, issued = 0;
    auto issue_next = [&]() {
        if (issued < total) {
            issue(nxt_tile, nxt_piece, nxt_stage);
            if (++nxt_piece == pieces) {
                nxt_piece = 0;
                ++nxt_tile;
            }
            nxt_stage = nxt_stage + 1 == kTalkStages ? 0 : nxt_stage + 1;
        }
        ++issued;
        cp_async_commit();      // an empty group keeps the count of groups in step
    };
#pragma unroll
    for (int i = 0; i < kTalkStages - 1; ++i) issue_next();

    int rpos[4], rwnd[4];       // the thread's rows: (block, half) -> 2 * block + half
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        rpos[i] = pos0 + (i >> 1) * 16 + (i & 1) * 8 + g;
        rwnd[i] = seq_row_window(rpos[i], p.window, p.chunk);
    }
    float m[4], l[4], o[2][kDvTiles][4], s[2][kKeys / 8][4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        m[i] = -INFINITY;
        l[i] = 0.0f;
    }
#pragma unroll
    for (int mt = 0; mt < 2; ++mt) {
#pragma unroll
        for (int nt = 0; nt < kDvTiles; ++nt) o[mt][nt][0] = o[mt][nt][1] = o[mt][nt][2] = o[mt][nt][3] = 0.0f;
#pragma unroll
        for (int nt = 0; nt < kKeys / 8; ++nt) s[mt][nt][0] = s[mt][nt][1] = s[mt][nt][2] = s[mt][nt][3] = 0.0f;
    }
    const float scale2 = p.scale * 1.4426950408889634f;    // the running softmax works in powers of two
    int st = 0;
    for (int it = 0; it < my_tiles; ++it) {
        for (int ip = 0; ip < pieces; ++ip) {
            cp_async_wait<kTalkStages - 2>();
            __syncthreads();        // the piece has landed for everyone, and everyone is done with the stage that is filled next
            issue_next();
            const uint32_t aQ = smem_u32(smh + st * stage_elems + warp * kBQ * kTalkCols), aK = smem_u32(smh + st * stage_elems + qrows * kTalkCols);
            st = st + 1 == kTalkStages ? 0 : st + 1;
#pragma unroll
            for (int ks = 0; ks < kTalkCols / 16; ++ks) {       // columns beyond the row are zeros in both operands
                uint32_t a0[4], a1[4];
                const uint32_t arow = (uint32_t)(lane & 15) * (kTalkCols * 2) + (uint32_t)(((2 * ks + (lane >> 4)) ^ (lane & 7)) << 4);
                ldmatrix_x4(a0, aQ + arow);
                ldmatrix_x4(a1, aQ + 16 * kTalkCols * 2 + arow);
#pragma unroll
                for (int np = 0; np < kKeys / 16; ++np) {
                    uint32_t bb[4];
                    const int row = np * 16 + (lane & 7) + ((lane >> 4) << 3);
                    ldmatrix_x4(bb, aK + (uint32_t)row * (kTalkCols * 2) + (uint32_t)(((2 * ks + ((lane >> 3) & 1)) ^ (lane & 7)) << 4));
                    mma_bf16_16816(s[0][2 * np], a0, bb[0], bb[1]);
                    mma_bf16_16816(s[0][2 * np + 1], a0, bb[2], bb[3]);
                    mma_bf16_16816(s[1][2 * np], a1, bb[0], bb[1]);
                    mma_bf16_16816(s[1][2 * np + 1], a1, bb[2], bb[3]);
                }
            }
        }
        // the tile's scores are complete: softmax, weighted values
        const int j0 = tiles.tile_of(split + it * p.nsplit) * kKeys;
        const uint32_t aV = smem_u32(smv + (it % v_bufs) * v_elems);
        // every key of the tile is seen by every query of the work item (interior of a window or chunk): no key is compared
        const bool inside = nq == kBQ && j0 + kKeys - 1 <= pos0 && last_pos - j0 < seq_row_window(last_pos, p.window, p.chunk);
#pragma unroll
        for (int mt = 0; mt < 2; ++mt) {
            float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
            for (int nt = 0; nt < kKeys / 8; ++nt) {
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int i = 2 * mt + (e >> 1), key = j0 + nt * 8 + 2 * c + (e & 1);
                    const float sc = s[mt][nt][e] * scale2;
                    s[mt][nt][e] = inside || seq_sees(rpos[i], key, rwnd[i], p.keep_first) ? sc : -INFINITY;
                    mx[e >> 1] = fmaxf(mx[e >> 1], s[mt][nt][e]);
                }
            }
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
                const int i = 2 * mt + hf;
                mx[hf] = fmaxf(mx[hf], __shfl_xor_sync(0xffffffffu, mx[hf], 1));
                mx[hf] = fmaxf(mx[hf], __shfl_xor_sync(0xffffffffu, mx[hf], 2));
                const float mn = fmaxf(m[i], mx[hf]);
                const float ref = mn == -INFINITY ? 0.0f : mn;        // no key seen yet: every weight below is 2^-inf = 0
                const float corr = fast_exp2(m[i] - ref);
                m[i] = mn;
                float sum = 0.0f;
#pragma unroll
                for (int nt = 0; nt < kKeys / 8; ++nt) {
#pragma unroll
                    for (int e = 2 * hf; e < 2 * hf + 2; ++e) {
                        s[mt][nt][e] = fast_exp2(s[mt][nt][e] - ref);
                        sum += s[mt][nt][e];
                    }
                }
                l[i] = l[i] * corr + sum;      // this thread's share of the row's sum; the quad's shares are added at the end
#pragma unroll
                for (int nt = 0; nt < kDvTiles; ++nt) {
                    o[mt][nt][2 * hf] *= corr;
                    o[mt][nt][2 * hf + 1] *= corr;
                }
            }
        }
#pragma unroll
        for (int ks = 0; ks < kKeys / 16; ++ks) {
            uint32_t ah[2][4], al[2][4];
#pragma unroll
            for (int mt = 0; mt < 2; ++mt) {
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    split_bf16(s[mt][2 * ks + half][0], s[mt][2 * ks + half][1], &ah[mt][2 * half], &al[mt][2 * half]);
                    split_bf16(s[mt][2 * ks + half][2], s[mt][2 * ks + half][3], &ah[mt][2 * half + 1], &al[mt][2 * half + 1]);
                }
            }
            const uint32_t vrow = aV + (uint32_t)((ks * 16 + (lane & 15)) * ldv + ((lane >> 4) << 3)) * 2;
#pragma unroll
            for (int nt = 0; nt < kDvTiles; nt += 2) {
                if (nt < dvt) {          // with an odd number of value tiles the last pair's second half is padding, and dropped
                    uint32_t bb[4];
                    ldmatrix_x4_trans(bb, vrow + nt * 16);
                    mma_bf16_16816(o[0][nt], ah[0], bb[0], bb[1]);
                    mma_bf16_16816(o[0][nt + 1], ah[0], bb[2], bb[3]);
                    mma_bf16_16816(o[1][nt], ah[1], bb[0], bb[1]);
                    mma_bf16_16816(o[1][nt + 1], ah[1], bb[2], bb[3]);
                    mma_bf16_16816(o[0][nt], al[0], bb[0], bb[1]);
                    mma_bf16_16816(o[0][nt + 1], al[0], bb[2], bb[3]);
                    mma_bf16_16816(o[1][nt], al[1], bb[0], bb[1]);
                    mma_bf16_16816(o[1][nt + 1], al[1], bb[2], bb[3]);
                }
            }
        }
#pragma unroll
        for (int mt = 0; mt < 2; ++mt)
#pragma unroll
            for (int nt = 0; nt < kKeys / 8; ++nt) s[mt][nt][0] = s[mt][nt][1] = s[mt][nt][2] = s[mt][nt][3] = 0.0f;
    }
    cp_async_wait<0>();
    const float snk = p.sink ? p.sink[h] : -INFINITY;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        l[i] += __shfl_xor_sync(0xffffffffu, l[i], 1);
        l[i] += __shfl_xor_sync(0xffffffffu, l[i], 2);
        const int r = (i >> 1) * 16 + (i & 1) * 8 + g, t = t0 + r;
        if (r >= nq) continue;
        m[i] *= 0.6931471805599453f;           // back to natural units (a share that saw no key stays at -inf)
        if (p.nsplit > 1) {
            float* rec = p.ws + (((size_t)t * p.heads + h) * p.nsplit + split) * (dv + 2);
            if (c == 0) {
                rec[0] = m[i];
                rec[1] = l[i];
            }
#pragma unroll
            for (int nt = 0; nt < kDvTiles; ++nt) {
                if (nt < dvt) {
                    rec[2 + nt * 8 + 2 * c] = o[i >> 1][nt][2 * (i & 1)];
                    rec[2 + nt * 8 + 2 * c + 1] = o[i >> 1][nt][2 * (i & 1) + 1];
                }
            }
            continue;
        }
        const float top = fmaxf(m[i], snk), w = expf(m[i] - top);
        const float inv = w / (l[i] * w + (p.sink ? expf(snk - top) : 0.0f));
        const size_t orow = (size_t)t * p.ldo + (size_t)h * dv, row16 = ((size_t)t * p.heads + h) * dv;
        const float* grow = p.gate ? p.gate + (size_t)t * p.ldg + (size_t)h * dv : nullptr;
#pragma unroll
        for (int nt = 0; nt < kDvTiles; ++nt) {
            if (nt < dvt) {
                const int col = nt * 8 + 2 * c;
                float v0 = o[i >> 1][nt][2 * (i & 1)] * inv, v1 = o[i >> 1][nt][2 * (i & 1) + 1] * inv;
                if (grow) {
                    v0 *= seq_sigmoid(grow[col]);
                    v1 *= seq_sigmoid(grow[col + 1]);
                }
                if (p.out) {
                    p.out[orow + col] = v0;
                    p.out[orow + col + 1] = v1;
                }
                if (p.out16) *reinterpret_cast<uint32_t*>(p.out16 + row16 + col) = pack_bf16(v0, v1);
            }
        }
    }
}

// ---- any size, fp32 or bf16 ----------------------------------------------------------------------------------------------------------------
constexpr int kTalkWarps = 8, kTalkHeads = 4;   // warps per CTA; query heads a warp scores (and weighs values for) at once

// shared memory of one CTA in bytes; the order of the parts in the kernel is the order here
__host__ __device__ inline size_t talk_smem(int nq, int gs, int heads, int dkq, int dv, int ldk, int ldv, int elem, int talk_in_smem) {
    const size_t floats = (talk_in_smem ? ((size_t)heads * heads + 3) / 4 * 4 : 0) + (size_t)nq * heads * dkq + ((size_t)nq * heads * dv + 3) / 4 * 4 +
                          2 * (size_t)nq * heads * kBK + ((size_t)3 * nq * heads + 3) / 4 * 4;
    return floats * sizeof(float) + (size_t)gs * kBK * (ldk + ldv) * elem;
}

template <typename KV>
__global__ void __launch_bounds__(kTalkWarps * 32) seq_attention_talk_kernel(TalkArgs p) {
    extern __shared__ __align__(16) float sm[];
    const int H = p.heads, G = p.kv_heads, group = H / G, dk = p.dk, dv = p.dv, NQ = p.nq;
    float* sT = sm;                                                                  // [H][H]
    float* sq = sT + (p.talk_in_smem ? ((size_t)H * H + 3) / 4 * 4 : 0);              // [NQ][H][dkq]
    float* so = sq + (size_t)NQ * H * p.dkq;                                          // [NQ][H][dv] unnormalised results
    float* ss = so + ((size_t)NQ * H * dv + 3) / 4 * 4;                               // [NQ][H][32] every head's own scores
    float* sp = ss + (size_t)NQ * H * kBK;                                            // [NQ][H][32] weights
    float* s_m = sp + (size_t)NQ * H * kBK;                                           // running maximum, sum, correction per (query, head)
    float* s_l = s_m + NQ * H;
    float* s_c = s_l + NQ * H;
    KV* sk = reinterpret_cast<KV*>(s_m + ((size_t)3 * NQ * H + 3) / 4 * 4);           // [gs][32][ldk]
    KV* sv = sk + (size_t)p.gs * kBK * p.ldk;                                         // [gs][32][ldv]
    const sllm_seq_batch& b = p.b;
    const int per_tile = kBQ / NQ, qt = b.T == b.nseg ? blockIdx.x : blockIdx.x / per_tile, sub = b.T == b.nseg ? 0 : blockIdx.x % per_tile;
    const int split = blockIdx.y, seg = b.qt_seg[qt], off = b.qt_off[qt] + sub * NQ;
    const int n = min(NQ, b.seg_len[seg] - off);
    if (n <= 0) return;
    const int t0 = b.seg_start[seg] + off, pos0 = b.seg_pos0[seg] + off, slot = b.seg_slot[seg], last_pos = pos0 + n - 1;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const KV* kp = reinterpret_cast<const KV*>(p.k_pool);
    const KV* vp = reinterpret_cast<const KV*>(p.v_pool);
    constexpr int E = 16 / sizeof(KV);
    const bool vec_k = dk % E == 0, vec_v = dv % E == 0;
    const TileList tiles(pos0, last_pos, seq_row_window(pos0, p.window, p.chunk), p.keep_first, kBK);

    // rows of key heads u0 .. u0 + ng - 1 (values: one head after the other in the pool) of tile j0; rows that do not exist are zeros
    auto stage = [&](bool keys, int j0, int u0, int ng) {
        const int page = b.block_table[(size_t)slot * b.max_pages + j0 / b.page_len], in_page = j0 % b.page_len, valid = min(kBK, last_pos + 1 - j0);
        const int width = keys ? dk : dv, ld = keys ? p.ldk : p.ldv;
        const KV* pool = keys ? kp : vp;
        KV* dst = keys ? sk : sv;
        auto row_of = [&](int u, int r) {
            return keys ? ((size_t)page * b.page_len + in_page + r) * G * dk + (size_t)u * dk : seq_pool_row(page, G, u, b.page_len, in_page + r, dv);
        };
        if (keys ? vec_k : vec_v) {
            const int units = width / E;
            for (int i = threadIdx.x; i < ng * kBK * units; i += blockDim.x) {
                const int un = i % units, r = (i / units) % kBK, u = i / (units * kBK);
                cp_async16(dst + ((size_t)u * kBK + r) * ld + un * E, r < valid ? pool + row_of(u0 + u, r) + un * E : pool, r < valid ? 16 : 0);
            }
        } else {
            for (int i = threadIdx.x; i < ng * kBK * ld; i += blockDim.x) {
                const int cc = i % ld, r = (i / ld) % kBK, u = i / (ld * kBK);
                dst[i] = r < valid && cc < width ? pool[row_of(u0 + u, r) + cc] : (KV)0;
            }
        }
        cp_async_commit();
    };

    if (split < tiles.n) {      // the first tile travels while the queries are fetched
        const int j0 = tiles.tile_of(split) * kBK;
        stage(true, j0, 0, min(p.gs, G));
        if (p.gs >= G) stage(false, j0, 0, G);
    }
    if (p.talk_in_smem)
        for (int i = threadIdx.x; i < H * H; i += blockDim.x) sT[i] = p.talk[i];
    const float* tm = p.talk_in_smem ? sT : p.talk;
    for (int i = threadIdx.x; i < NQ * H * p.dkq; i += blockDim.x) {
        const int cc = i % p.dkq, h = (i / p.dkq) % H, r = i / (p.dkq * H);
        sq[i] = r < n && cc < dk ? p.q[(size_t)(t0 + r) * p.ldq + (size_t)h * dk + cc] : 0.0f;
    }
    for (int i = threadIdx.x; i < NQ * H * dv; i += blockDim.x) so[i] = 0.0f;
    for (int i = threadIdx.x; i < NQ * H; i += blockDim.x) {
        s_m[i] = -INFINITY;
        s_l[i] = 0.0f;
    }
    // heads of a group a warp takes at once: fewer when that leaves warps without work
    int hb = kTalkHeads;
    while (hb > 1 && n * min(p.gs, G) * ((group + hb - 1) / hb) < kTalkWarps) hb >>= 1;
    const int hblocks = (group + hb - 1) / hb, cblocks = (dv + 63) / 64;
    int hv = kTalkHeads;
    while (hv > 1 && n * min(p.gs, G) * ((group + hv - 1) / hv) * cblocks < kTalkWarps) hv >>= 1;
    const int vblocks = (group + hv - 1) / hv;
    bool first = true;
    for (int idx = split; idx < tiles.n; idx += p.nsplit) {
        const int j0 = tiles.tile_of(idx) * kBK, valid = min(kBK, last_pos + 1 - j0);
        for (int u0 = 0; u0 < G; u0 += p.gs) {
            const int ng = min(p.gs, G - u0);
            if (!first) {
                __syncthreads();            // everyone is done with the stages
                stage(true, j0, u0, ng);
                if (p.gs >= G) stage(false, j0, 0, G);
            }
            first = false;
            if (p.gs >= G) cp_async_wait<1>();   // the keys are here; the values may still travel
            else cp_async_wait<0>();
            __syncthreads();
            for (int it = warp; it < n * ng * hblocks; it += kTalkWarps) {
                const int hbl = it % hblocks, u = (it / hblocks) % ng, r = it / (hblocks * ng);
                const int hh0 = hbl * hb, nh = min(hb, group - hh0), h0 = (u0 + u) * group + hh0;
                const KV* krow = sk + ((size_t)u * kBK + lane) * p.ldk;
                const float* qrow = sq + ((size_t)r * H + h0) * p.dkq;
                float acc[kTalkHeads] = {0.0f, 0.0f, 0.0f, 0.0f};
                for (int cc = 0; cc < dk; cc += E) {
                    float kv[E];
                    seq_ld16(krow + cc, true, kv);
#pragma unroll
                    for (int x = 0; x < kTalkHeads; ++x) {
                        if (x < nh) {
#pragma unroll
                            for (int e = 0; e < E; e += 4) {
                                const float4 qv = *reinterpret_cast<const float4*>(qrow + (size_t)x * p.dkq + cc + e);
                                acc[x] = fmaf(qv.x, kv[e], acc[x]);
                                acc[x] = fmaf(qv.y, kv[e + 1], acc[x]);
                                acc[x] = fmaf(qv.z, kv[e + 2], acc[x]);
                                acc[x] = fmaf(qv.w, kv[e + 3], acc[x]);
                            }
                        }
                    }
                }
#pragma unroll
                for (int x = 0; x < kTalkHeads; ++x)
                    if (x < nh) ss[((size_t)r * H + h0 + x) * kBK + lane] = acc[x] * p.scale;
            }
        }
        __syncthreads();
        // the heads' scores mixed, and the running softmax of every (query, head): lane = key
        for (int it = warp; it < n * H; it += kTalkWarps) {
            const int h = it % H, r = it / H, qpos = pos0 + r;
            const float* own = ss + (size_t)r * H * kBK + lane;
            float sc = 0.0f;
#pragma unroll 4
            for (int x = 0; x < H; ++x) sc = fmaf(tm[(size_t)h * H + x], own[(size_t)x * kBK], sc);
            const bool see = seq_sees(qpos, j0 + lane, seq_row_window(qpos, p.window, p.chunk), p.keep_first);
            sc = see ? sc : -INFINITY;
            const float old = s_m[it], mn = fmaxf(old, warp_max(sc));
            const float w = see ? expf(sc - mn) : 0.0f, sum = warp_sum(w);
            sp[(size_t)it * kBK + lane] = w;
            __syncwarp();
            if (lane == 0) {
                const float corr = mn == -INFINITY ? 1.0f : expf(old - mn);
                s_m[it] = mn;
                s_l[it] = s_l[it] * corr + sum;
                s_c[it] = corr;
            }
        }
        for (int u0 = 0; u0 < G; u0 += p.gs) {
            const int ng = min(p.gs, G - u0);
            if (p.gs < G) {
                __syncthreads();
                stage(false, j0, u0, ng);
            }
            cp_async_wait<0>();
            __syncthreads();
            for (int it = warp; it < n * ng * vblocks * cblocks; it += kTalkWarps) {
                const int cb = it % cblocks, vb = (it / cblocks) % vblocks, u = (it / (cblocks * vblocks)) % ng, r = it / (cblocks * vblocks * ng);
                const int hh0 = vb * hv, nh = min(hv, group - hh0), h0 = (u0 + u) * group + hh0;
                const int c0 = cb * 64 + lane, c1 = c0 + 32;
                const KV* vcol = sv + (size_t)u * kBK * p.ldv;
                const float* prow = sp + ((size_t)r * H + h0) * kBK;
                float a0[kTalkHeads] = {0.0f, 0.0f, 0.0f, 0.0f}, a1[kTalkHeads] = {0.0f, 0.0f, 0.0f, 0.0f};
                for (int j = 0; j < valid; j += 4) {     // weights and values beyond `valid` are zeros
                    float v0[4], v1[4];
#pragma unroll
                    for (int x = 0; x < 4; ++x) {
                        v0[x] = c0 < dv ? seq_ld(vcol, (size_t)(j + x) * p.ldv + c0) : 0.0f;
                        v1[x] = c1 < dv ? seq_ld(vcol, (size_t)(j + x) * p.ldv + c1) : 0.0f;
                    }
#pragma unroll
                    for (int x = 0; x < kTalkHeads; ++x) {
                        if (x < nh) {
                            const float4 w = *reinterpret_cast<const float4*>(prow + (size_t)x * kBK + j);
                            a0[x] = fmaf(w.x, v0[0], fmaf(w.y, v0[1], fmaf(w.z, v0[2], fmaf(w.w, v0[3], a0[x]))));
                            a1[x] = fmaf(w.x, v1[0], fmaf(w.y, v1[1], fmaf(w.z, v1[2], fmaf(w.w, v1[3], a1[x]))));
                        }
                    }
                }
#pragma unroll
                for (int x = 0; x < kTalkHeads; ++x) {
                    if (x < nh) {
                        const float corr = s_c[r * H + h0 + x];
                        float* orow = so + ((size_t)r * H + h0 + x) * dv;
                        if (c0 < dv) orow[c0] = fmaf(orow[c0], corr, a0[x]);
                        if (c1 < dv) orow[c1] = fmaf(orow[c1], corr, a1[x]);
                    }
                }
            }
        }
    }
    cp_async_wait<0>();
    __syncthreads();
    for (int it = warp; it < n * H; it += kTalkWarps) {
        const int h = it % H, r = it / H;
        float* rec = p.ws + (((size_t)(t0 + r) * H + h) * p.nsplit + split) * (dv + 2);
        if (lane == 0) {
            rec[0] = s_m[it];
            rec[1] = s_l[it];
        }
        for (int cc = lane; cc < dv; cc += 32) rec[2 + cc] = so[(size_t)it * dv + cc];
    }
}

}  // namespace sllm

using namespace sllm;

extern "C" {

int sllm_seq_attention_talk_takes_mixed(int32_t heads, int32_t kv_heads, int32_t dk, int32_t dv, int32_t kv_dtype) {
    return kv_dtype == SLLM_BF16 && heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && (kv_heads * dk) % 8 == 0 && dv % 8 == 0 && dv <= 128 && g_tune_seq_attn_mma;
}

int sllm_seq_attention_talk(const sllm_seq_batch* b, const float* q, int32_t ldq, const void* q_mixed, int32_t heads, int32_t kv_heads, int32_t dk, int32_t dv,
                            float scale, const float* talk, const void* k_pool, const void* v_pool, int32_t kv_dtype, int32_t nsplit, float* ws,
                            const sllm_seq_attn_opts* opts, const float* gate, int32_t ldg, const float* sink, float* out, int32_t ldo, void* out16,
                            sllm_stream_t stream) {
    SLLM_REQUIRE(b && b->T > 0 && b->nseg > 0 && b->tok_slot && b->tok_pos && b->seg_start && b->seg_len && b->seg_slot && b->seg_pos0 && b->block_table &&
                 b->qt_seg && b->qt_off && b->n_qtiles > 0, SLLM_EINVAL, "seq_attention_talk: incomplete batch description");
    SLLM_REQUIRE((q || q_mixed) && talk && k_pool && v_pool && (out || out16), SLLM_EINVAL, "seq_attention_talk: bad argument");
    SLLM_REQUIRE(heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dk > 0 && dv > 0, SLLM_EINVAL, "seq_attention_talk: %d query heads over %d kv heads", heads, kv_heads);
    SLLM_REQUIRE(!opts || (opts->window >= 0 && opts->keep_first >= 0 && opts->chunk >= 0 && !(opts->window && opts->chunk)), SLLM_EINVAL,
                 "seq_attention_talk: a window or chunks, not both");
    SLLM_REQUIRE(!opts || (opts->softcap == 0.0f && !opts->slopes && !opts->logdist && !opts->values_in_keys && !opts->cross_values), SLLM_ENOTSUP,
                 "seq_attention_talk: only windows and chunks");
    SLLM_REQUIRE(b->page_len % kBK == 0, SLLM_ENOTSUP, "seq_attention_talk: pages of a multiple of %d positions", kBK);
    SLLM_REQUIRE(nsplit >= 1 && nsplit <= 8192, SLLM_EINVAL, "seq_attention_talk: nsplit");
    SLLM_REQUIRE(kv_dtype == SLLM_F32 || kv_dtype == SLLM_BF16, SLLM_ENOTSUP, "seq_attention_talk: fp32 or bf16 pools");
    cudaStream_t st = as_stream(stream);
    TalkArgs p{};
    p.b = *b; p.q = q; p.ldq = ldq; p.qm = (const uint16_t*)q_mixed; p.heads = heads; p.kv_heads = kv_heads; p.dk = dk; p.dv = dv; p.scale = scale; p.talk = talk;
    p.k_pool = k_pool; p.v_pool = v_pool; p.nsplit = nsplit; p.ws = ws;
    p.window = opts && opts->window > 0 ? opts->window : INT_MAX;
    p.keep_first = opts && opts->window > 0 ? opts->keep_first : 0;
    p.chunk = opts ? opts->chunk : 0;
    p.sink = sink; p.gate = gate; p.ldg = ldg; p.out = out; p.ldo = ldo; p.out16 = (uint16_t*)out16;
    if (q_mixed) {
        SLLM_REQUIRE(sllm_seq_attention_talk_takes_mixed(heads, kv_heads, dk, dv, kv_dtype), SLLM_ENOTSUP, "seq_attention_talk: mixed queries for heads of %d + %d", dk, dv);
        SLLM_REQUIRE(nsplit == 1 || ws, SLLM_EINVAL, "seq_attention_talk: %d shares need a workspace", nsplit);
        const int group = heads / kv_heads, hpc = group % 4 == 0 ? 4 : (group % 2 == 0 ? 2 : 1), pieces = (kv_heads * dk + kTalkCols - 1) / kTalkCols;
        const dim3 grid(b->n_qtiles, heads / hpc, nsplit);
        const size_t smem = (kTalkStages * (size_t)(hpc * kBQ + kTalkKeys) * kTalkCols + (size_t)(pieces == 1 ? 3 : 2) * kTalkKeys * (dv + 8)) * sizeof(uint16_t);
#define SLLM_TALK_LAUNCH(DV, HEADS)                                                                                                                    \
    do {                                                                                                                                               \
        SLLM_CUDA(cudaFuncSetAttribute(seq_attention_talk_mma_kernel<DV, HEADS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));             \
        seq_attention_talk_mma_kernel<DV, HEADS><<<grid, 32 * HEADS, smem, st>>>(p);                                                                   \
    } while (0)
        if (dv <= 64) {
            if (hpc == 4) SLLM_TALK_LAUNCH(8, 4); else if (hpc == 2) SLLM_TALK_LAUNCH(8, 2); else SLLM_TALK_LAUNCH(8, 1);
        } else {
            if (hpc == 4) SLLM_TALK_LAUNCH(16, 4); else if (hpc == 2) SLLM_TALK_LAUNCH(16, 2); else SLLM_TALK_LAUNCH(16, 1);
        }
#undef SLLM_TALK_LAUNCH
        ++g_launches;
        SLLM_LAUNCH_CHECK();
        if (nsplit == 1) return SLLM_OK;
        return launch_attention_finish(b, ws, nsplit, heads, dv, nullptr, 0, gate, ldg, 1, sink, out, ldo, (uint16_t*)out16, st);
    }
    SLLM_REQUIRE(ws, SLLM_EINVAL, "seq_attention_talk: no workspace");
    // geometry: as many queries per CTA and as many heads per stage as shared memory takes (single tokens: one query per CTA)
    const int elem = kv_dtype == SLLM_BF16 ? 2 : 4, E = 16 / elem;
    auto odd_units = [&](int w) { const int u = (w + E - 1) / E; return (u | 1) * E; };     // row length of an odd number of 16-byte units: no bank conflicts
    p.dkq = (dk + 7) & ~7;
    p.ldk = odd_units(dk);
    p.ldv = (dv + E - 1) / E * E;
    const size_t budget = (size_t)smem_optin_bytes() - 1024;
    p.talk_in_smem = talk_smem(1, 1, heads, p.dkq, dv, p.ldk, p.ldv, elem, 1) <= budget;
    SLLM_REQUIRE(talk_smem(1, 1, heads, p.dkq, dv, p.ldk, p.ldv, elem, p.talk_in_smem) <= budget, SLLM_ENOTSUP,
                 "seq_attention_talk: %d heads of %d + %d do not fit shared memory", heads, dk, dv);
    p.nq = b->T == b->nseg ? 1 : 4;
    while (p.nq > 1 && talk_smem(p.nq, 1, heads, p.dkq, dv, p.ldk, p.ldv, elem, p.talk_in_smem) > budget) p.nq >>= 1;
    p.gs = kv_heads;
    while (p.gs > 1 && talk_smem(p.nq, p.gs, heads, p.dkq, dv, p.ldk, p.ldv, elem, p.talk_in_smem) > budget) --p.gs;
    const size_t smem = talk_smem(p.nq, p.gs, heads, p.dkq, dv, p.ldk, p.ldv, elem, p.talk_in_smem);
    const dim3 grid(b->T == b->nseg ? b->n_qtiles : b->n_qtiles * (kBQ / p.nq), nsplit);
    if (kv_dtype == SLLM_F32) {
        SLLM_CUDA(cudaFuncSetAttribute(seq_attention_talk_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        seq_attention_talk_kernel<float><<<grid, kTalkWarps * 32, smem, st>>>(p);
    } else {
        SLLM_CUDA(cudaFuncSetAttribute(seq_attention_talk_kernel<uint16_t>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        seq_attention_talk_kernel<uint16_t><<<grid, kTalkWarps * 32, smem, st>>>(p);
    }
    ++g_launches;
    SLLM_LAUNCH_CHECK();
    return launch_attention_finish(b, ws, nsplit, heads, dv, nullptr, 0, gate, ldg, 1, sink, out, ldo, (uint16_t*)out16, st);
}

}  // extern "C"
