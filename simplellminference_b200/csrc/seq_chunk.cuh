// csrc/seq_chunk.cuh — the recurrences of seq_delta.cu in blocks of 16 tokens on the tensor cores (seq_chunk.cu): arguments and launch.
#pragma once
#include "seq_common.cuh"

namespace sllm {

constexpr int kChunk = 16;          // tokens of a block
constexpr int kChunkMaxKey = 128;   // key channels of a head, at most

struct ChunkArgs {
    sllm_seq_batch b;
    const float *q, *k, *v; int ldq, ldk, ldv;
    int delta;                                           // 1: delta rule; 0: linear attention with a constant decay
    // delta rule: logits of beta [heads] and of the decay's step ([heads], or [heads * dk] with `channel`), A_log [heads], dt_bias like the step
    const float *bl, *al; int ldb, lda; const float *A_log, *dt_bias; int channel;
    // constant decay: [heads] minus the decay's logarithm; (cos, sin) [T][n_freq] that turn q and k (NULL = not); q, k and v pass silu
    const float* rate; const float2* angles; int n_freq, layout, silu;
    int heads, kv_heads, dk, dv;
    float unit_eps, scale;                               // delta rule: q times scale; constant decay: k times scale
    float* state; float* o; int ldo;
    uint8_t* ws;                                         // chunk_ws_bytes: the blocks' records, then
    float* v_ws;                                         // values passed through silu [blocks][16][heads * dv] (set by the launch)
};

// key channels rounded up to what the kernel is instantiated for
__host__ __device__ __forceinline__ int chunk_key(int dk) { return dk <= 32 ? 32 : dk <= 64 ? 64 : dk <= 96 ? 96 : 128; }
// per block and head: decayed keys, decayed queries and keys decayed to the block's end as (hi, lo) bf16 fragments, the two 16 x 16 matrices
// likewise, the block's decay per key channel
__host__ __device__ constexpr size_t chunk_record_bytes(int dkp) { return (size_t)dkp * (6 * kChunk * 2 + 4) + 4 * kChunk * kChunk * 2; }
inline size_t chunk_ws_bytes(int n_qtiles, int heads, int dk, int dv) {
    return 2 * (size_t)n_qtiles * heads * (chunk_record_bytes(chunk_key(dk)) + (size_t)kChunk * dv * sizeof(float));
}
int launch_chunk_scan(const ChunkArgs& p, cudaStream_t st);

}  // namespace sllm
