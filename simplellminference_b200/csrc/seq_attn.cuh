// csrc/seq_attn.cuh — what the attention kernels of the ragged token batch share (seq_attn.cu, seq_attn_talk.cu): tile sizes, which keys a
// query sees and which key tiles a CTA visits, the bf16 tensor-core product and its operand packing, asynchronous copies.
#pragma once
#include <climits>

#include "seq_common.cuh"

namespace sllm {

constexpr int kBQ = 32, kBK = 32;   // queries per attention work item (the engine's query tiles), keys per tile

// Launches the merge of the shares (seq_attn.cu); arguments as sllm_seq_attention_finish.
int launch_attention_finish(const sllm_seq_batch* b, const float* ws, int nsplit, int heads, int dv, const double* vfreq, int layout, const float* gate, int ldg,
                            int gate_channels, const float* sink, float* out, int ldo, uint16_t* out16, cudaStream_t st);

#ifdef __CUDACC__

// The key tiles a CTA whose queries lie at positions first .. last has to visit: the tiles of the kept first positions, then the tiles
// from the one that holds the oldest key inside the first query's window up to the last query's own tile.
struct TileList {
    int n_keep, lo, n;
    __device__ __forceinline__ TileList(int first, int last, int window, int keep_first, int tile) {
        const int nkt = last / tile + 1;
        const int oldest = window > first ? 0 : first - window + 1;
        lo = oldest / tile;
        n_keep = min(lo, (min(keep_first, oldest) + tile - 1) / tile);
        n = n_keep + nkt - lo;
    }
    __device__ __forceinline__ int tile_of(int idx) const { return idx < n_keep ? idx : lo + idx - n_keep; }
};

// How far back the query at `qpos` sees, itself included: a sliding window of fixed size, or, with chunks of positions counted from the
// sequence's start, back to the first position of the query's own chunk.
__device__ __forceinline__ int seq_row_window(int qpos, int window, int chunk) { return chunk > 0 ? qpos % chunk + 1 : window; }
__device__ __forceinline__ bool seq_sees(int qpos, int key, int window, int keep_first) {
    return key <= qpos && (qpos - key < window || key < keep_first);
}


__device__ __forceinline__ void mma_bf16_16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// p = hi + lo with both terms bf16: hi = round(p), lo = round(p - hi)
__device__ __forceinline__ void split_bf16(float p0, float p1, uint32_t* hi, uint32_t* lo) {
    const uint32_t h = pack_bf16(p0, p1);
    *hi = h;
    *lo = pack_bf16(p0 - __uint_as_float(h << 16), p1 - __uint_as_float(h & 0xffff0000u));
}

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
// 16 bytes global -> shared without passing through registers; bytes = 0 writes zeros and reads nothing
__device__ __forceinline__ void cp_async16(void* dst, const void* src, int bytes) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

#endif

}  // namespace sllm
