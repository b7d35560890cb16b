// Pieces that recurrences in chunks of 64 tokens share: ldmatrix / mma.sync fragments, and floats that go into a tensor-core
// product as two bfloat16 terms.
#pragma once

#include "common.cuh"

#define CM_CHUNK 64
#define CM_PAD 8             // bfloat16 values between rows in shared memory: ldmatrix reads eight rows without bank conflicts

__device__ __forceinline__ uint32_t cm_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cm_ldm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void cm_ldm4t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void cm_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t cm_pack(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&v);
}
// a pair of floats as two bfloat16 pairs: the rounding, and what it left
__device__ __forceinline__ void cm_split(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const float2 f = __bfloat1622float2(h);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = cm_pack(x - f.x, y - f.y);
}

// chunks a step can have at most (every sequence may end in a partial chunk)
static inline int cm_max_chunks(int n_tokens, int n_seqs) {
    const int by_tokens = n_tokens / CM_CHUNK + n_seqs;
    return by_tokens < n_tokens ? by_tokens : n_tokens;
}

// chunk number `idx` of the step -> its sequence and its first token there; false beyond the step's last chunk
__device__ __forceinline__ bool cm_find_chunk(const int* __restrict__ seq_start, const int* __restrict__ tok_pos, int n_seqs, int idx, int& seq, int& t0) {
    for (int s = 0; s < n_seqs; ++s) {
        const int n = seq_start[s + 1] - seq_start[s];
        const int nc = (n > 0 && tok_pos[seq_start[s]] >= 0) ? (n + CM_CHUNK - 1) / CM_CHUNK : 0;
        if (idx < nc) { seq = s; t0 = idx * CM_CHUNK; return true; }
        idx -= nc;
    }
    return false;
}

// CM_CHUNK rows of `width` bfloat16 values (a multiple of 8) from packed rows into shared memory, 16 bytes a copy; rows from L on are zeros
__device__ __forceinline__ void cm_fill(__nv_bfloat16* dst, int dst_stride, const __nv_bfloat16* src, long long src_stride, int width, int L, int tid, int threads) {
    const int per = width >> 3;
    for (int idx = tid; idx < CM_CHUNK * per; idx += threads) {
        const int j = idx / per, c = (idx - j * per) << 3;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (j < L) v = *reinterpret_cast<const uint4*>(src + (long long)j * src_stride + c);
        *reinterpret_cast<uint4*>(dst + j * dst_stride + c) = v;
    }
}
