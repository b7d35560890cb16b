// The matrix memory in chunks, for many tokens in bfloat16 (the equations and the token-by-token form are matrix_memory.cu's).
//
// Without the running maximum the recurrence is S~_t = e^f S~_(t-1) + e^i k v^T, and S_t = e^(-m_t) S~_t with
// m_t = max(f + m_(t-1), i).  With chunks of 64 tokens, S, n and m those before a chunk's first token, L its tokens, i and j
// places inside it, all logarithms to base two, c_i the sum of the forget gates up to i and g_i = max_(j <= i) (in_j - c_j):
//   m_i  = c_i + max(m, g_i)
//   P_ij = (q_i . k_j) 2^(c_i - c_j + in_j - m_i) for j <= i,     w_i = 2^(c_i + m - m_i)
//   o_i  = (sum_j P_ij v_j + w_i S^T q_i) / (max(|sum_j P_ij + w_i n . q_i|, 2^(-m_i)) + den_eps)
//   A    = max_j (c_(L-1) - c_j + in_j),   U = sum_j k_j (2^(c_(L-1) - c_j + in_j - A) v_j)^T,   u likewise without v
//   m'   = max(c_(L-1) + m, A),   S' = 2^(c_(L-1) + m - m') S + 2^(A - m') U,   n' likewise with u.
// No exponent is above zero.  U, u, c and A need nothing of the chunks before, and o needs of them only S, n and m, so the
// work is parallel over chunks in three launches, as for the state space (state_space_chunked.cu):
//   1. mm_chunk_kernel<false>: a block per (chunk, head, 64 state columns): U on tensor cores, u, c_(L-1) and A;
//   2. mm_scan_kernel: a thread per four elements of S (and of n) walks its sequence's chunks in float, leaving in the work
//      buffer what stands BEFORE each chunk and in the cache what stands after the last;
//   3. mm_chunk_kernel<true>: the outputs.
// q, k and v are bfloat16 as the projection left them (exact operands).  The weighted v of step 1, P and S go into their
// products as two bfloat16 terms (16 bits of them count); every sum is float, and so are the gates and their exponentials.
#include "api.h"
#include "chunk_mma.cuh"
#include "common.cuh"
#include "launch.cuh"
#include "matrix_memory.cuh"

namespace {

#define MMC_COLS 64
#define MMC_THREADS 256

struct ChunkWork {
    float* totals;      // [chunks][heads][2]: c_(L-1) and A
    float* m_before;    // [chunks][heads]
    float* m_first;     // [seqs][heads]: m before the step
    float* n_work;      // [chunks][heads][dim]: u, then n before the chunk
    float* s_work;      // [chunks][heads][dim][vdim]: U, then S before the chunk
};

template <bool OUTPUT>
__global__ void __launch_bounds__(MMC_THREADS) mm_chunk_kernel(MatrixMemoryArgs a, ChunkWork work) {
    extern __shared__ __align__(16) unsigned char mmc_raw[];
    const int dim = a.dim, vdim = a.vdim;
    const int h = blockIdx.y, c0 = blockIdx.z * MMC_COLS;
    const int nv = min(MMC_COLS, vdim - c0);               // columns of this block (a multiple of 16)
    const int qs = dim + CM_PAD, vs = MMC_COLS + CM_PAD;    // row strides in shared memory, in values
    __nv_bfloat16* Ks = reinterpret_cast<__nv_bfloat16*>(mmc_raw);    // [64][qs]
    __nv_bfloat16* Vh = Ks + CM_CHUNK * qs;                             // [64][vs]  v (OUTPUT), or the weighted v's rounding
    __nv_bfloat16* Vl = Vh + CM_CHUNK * vs;                             // [64][vs]  what that rounding left (not OUTPUT)
    __nv_bfloat16* Qs = Vl;                                             // [64][qs]  OUTPUT only, like the two below
    __nv_bfloat16* Sh = Qs + CM_CHUNK * qs;                             // [dim][vs] the state before the chunk, rounded
    __nv_bfloat16* Sl = Sh + dim * vs;                                  // [dim][vs] what the rounding left
    __shared__ float ig[CM_CHUNK], cl[CM_CHUNK], mi[CM_CHUNK], qn[CM_CHUNK];      // in_j, c_j, m_i, n . q_i
    __shared__ float n_s[128];
    int seq, t0;
    if (!cm_find_chunk(a.seq_start, a.tok_pos, a.n_seqs, blockIdx.x, seq, t0)) return;
    const int row0 = a.seq_start[seq], n = a.seq_start[seq + 1] - row0;
    const int L = min(CM_CHUNK, n - t0);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
    const int ksteps = dim >> 4, n_mt = dim >> 4, nt_count = nv >> 3;
    const __nv_bfloat16* rows = (const __nv_bfloat16*)a.rows + (long long)(row0 + t0) * a.row_stride;
    const long long ch = (long long)blockIdx.x * a.n_heads + h;
    float* W = work.s_work + ch * dim * vdim + c0;
    rdl_grid_wait();
    rdl_grid_launch_dependents();

    // the gates and the running sums and maxima: a warp, two tokens a lane, in token order
    if (warp == 0) {
        const float bi = a.i_bias[h], bf = a.f_bias[h];
        const float m = OUTPUT ? __ldcg(work.m_before + ch) : 0.f;
        const int j0 = 2 * lane, j1 = j0 + 1;
        float i0 = -INFINITY, i1 = -INFINITY, f0 = 0.f, f1 = 0.f;
        if (j0 < L) {
            i0 = mm_input_gate(__bfloat162float(rows[(long long)j0 * a.row_stride + a.i_col + h]), bi, a.cap);
            f0 = mm_forget_gate(__bfloat162float(rows[(long long)j0 * a.row_stride + a.f_col + h]), bf, a.cap);
        }
        if (j1 < L) {
            i1 = mm_input_gate(__bfloat162float(rows[(long long)j1 * a.row_stride + a.i_col + h]), bi, a.cap);
            f1 = mm_forget_gate(__bfloat162float(rows[(long long)j1 * a.row_stride + a.f_col + h]), bf, a.cap);
        }
        float run = f0 + f1;
#pragma unroll
        for (int off = 1; off < 32; off <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, run, off);
            if (lane >= off) run += up;
        }
        const float s0 = run - f1, s1 = run;               // c of the two tokens
        float best = fmaxf(i0 - s0, i1 - s1);               // places beyond the chunk's end: minus infinity
#pragma unroll
        for (int off = 1; off < 32; off <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, best, off);
            if (lane >= off) best = fmaxf(best, up);
        }
        const float before = __shfl_up_sync(0xffffffffu, best, 1);      // g of the tokens before this lane's
        const float g0 = fmaxf(lane > 0 ? before : -INFINITY, i0 - s0);
        ig[j0] = i0; ig[j1] = i1;
        cl[j0] = s0; cl[j1] = s1;
        if (OUTPUT) {
            mi[j0] = s0 + fmaxf(m, g0);
            mi[j1] = s1 + fmaxf(m, best);
        } else {
            const float c_end = __shfl_sync(0xffffffffu, run, 31);       // gates beyond the chunk's end are zero
            const float top = c_end + __shfl_sync(0xffffffffu, best, 31);
            if (lane == 0) {
                mi[0] = top;
                if (blockIdx.z == 0) {
                    work.totals[2 * ch] = c_end;
                    work.totals[2 * ch + 1] = top;
                    if (t0 == 0)
                        work.m_first[(long long)seq * a.n_heads + h] =
                            a.norm[((long long)a.slots[seq] * a.n_heads + h) * ((vdim + MM_COLS - 1) / MM_COLS) * (dim + 1) + dim];
                }
            }
        }
    }
    cm_fill(Ks, qs, rows + a.k_col + h * dim, a.row_stride, dim, L, tid, MMC_THREADS);
    if (OUTPUT) {
        cm_fill(Qs, qs, rows + a.q_col + h * dim, a.row_stride, dim, L, tid, MMC_THREADS);
        cm_fill(Vh, vs, rows + a.v_col + h * vdim + c0, a.row_stride, nv, L, tid, MMC_THREADS);
        for (int i = tid; i < dim; i += MMC_THREADS) n_s[i] = __ldcg(work.n_work + ch * dim + i);
        // the state before this chunk as two bfloat16 terms
#pragma unroll 4
        for (int idx = tid; idx < dim * (nv >> 2); idx += MMC_THREADS) {
            const int r = idx / (nv >> 2), c = 4 * (idx - r * (nv >> 2));
            const float4 sv = __ldcg(reinterpret_cast<const float4*>(W + (long long)r * vdim + c));
            uint2 hi, lo;
            cm_split(sv.x, sv.y, hi.x, lo.x);
            cm_split(sv.z, sv.w, hi.y, lo.y);
            *reinterpret_cast<uint2*>(Sh + r * vs + c) = hi;
            *reinterpret_cast<uint2*>(Sl + r * vs + c) = lo;
        }
    }
    __syncthreads();

    if (!OUTPUT) {
        // v_j 2^(c_(L-1) - c_j + in_j - A), as two terms
        const float c_end = cl[L - 1], top = mi[0];
        for (int idx = tid; idx < CM_CHUNK * (nv >> 1); idx += MMC_THREADS) {
            const int j = idx / (nv >> 1), c = 2 * (idx - j * (nv >> 1));
            uint32_t hi = 0u, lo = 0u;
            if (j < L) {
                const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(rows + (long long)j * a.row_stride + a.v_col + h * vdim + c0 + c));
                const float wj = exp2f(c_end - cl[j] + ig[j] - top);
                cm_split(v.x * wj, v.y * wj, hi, lo);
            }
            *reinterpret_cast<uint32_t*>(Vh + j * vs + c) = hi;
            *reinterpret_cast<uint32_t*>(Vl + j * vs + c) = lo;
        }
        if (blockIdx.z == 0) {
            if (tid < CM_CHUNK) qn[tid] = tid < L ? exp2f(c_end - cl[tid] + ig[tid] - top) : 0.f;
        }
        __syncthreads();
        if (blockIdx.z == 0) {
            for (int i = tid; i < dim; i += MMC_THREADS) {
                float u = 0.f;
                for (int j = 0; j < L; ++j) u = fmaf(qn[j], __bfloat162float(Ks[j * qs + i]), u);
                work.n_work[ch * dim + i] = u;
            }
        }
        // ---- U = K^T V_w: rows 16 warp .. + 15 of the state are this warp's ----
        if (warp < n_mt) {
            const int m0 = warp * 16;
            float u[8][4];
#pragma unroll
            for (int nt = 0; nt < 8; ++nt) u[nt][0] = u[nt][1] = u[nt][2] = u[nt][3] = 0.f;
#pragma unroll
            for (int kb = 0; kb < 4; ++kb) {
                uint32_t ka[4];
                cm_ldm4t(ka, cm_smem(Ks + (kb * 16 + ((lane >> 4) << 3) + (lane & 7)) * qs + m0 + (((lane >> 3) & 1) << 3)));
#pragma unroll
                for (int nb = 0; nb < 4; ++nb) {
                    if (2 * nb >= nt_count) continue;
                    const int off = (kb * 16 + (((lane >> 3) & 1) << 3) + (lane & 7)) * vs + nb * 16 + ((lane >> 4) << 3);
                    uint32_t bh[4], bl[4];
                    cm_ldm4t(bh, cm_smem(Vh + off));
                    cm_ldm4t(bl, cm_smem(Vl + off));
                    cm_mma(u[2 * nb], ka, bh[0], bh[1]);
                    cm_mma(u[2 * nb + 1], ka, bh[2], bh[3]);
                    cm_mma(u[2 * nb], ka, bl[0], bl[1]);
                    cm_mma(u[2 * nb + 1], ka, bl[2], bl[3]);
                }
            }
#pragma unroll
            for (int nt = 0; nt < 8; ++nt) {
                if (nt >= nt_count) continue;
#pragma unroll
                for (int hh = 0; hh < 2; ++hh)
                    *reinterpret_cast<float2*>(W + (long long)(m0 + g + 8 * hh) * vdim + nt * 8 + 2 * tq) = make_float2(u[nt][2 * hh], u[nt][2 * hh + 1]);
            }
        }
        return;
    }

    // n . q_i: four threads a row, every fourth pair of its values each
    {
        const int i = tid >> 2, part = tid & 3;
        float s = 0.f;
        for (int d = 2 * part; d < dim; d += 8) {
            const float2 qv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(Qs + i * qs + d));
            s = fmaf(qv.x, n_s[d], s);
            s = fmaf(qv.y, n_s[d + 1], s);
        }
        s += __shfl_xor_sync(0xffffffffu, s, 1);
        s += __shfl_xor_sync(0xffffffffu, s, 2);
        if (part == 0) qn[i] = s;
    }
    // ---- P, rows 16 rw .. + 15 ----
    // warps rw and rw + 4 share the rows 16 rw .. + 15 (each forms P for itself) and take 32 of the block's 64 columns each
    const int rw = warp & 3, cw = warp >> 2;
    const int i_hi = rw * 16 + g + 8;       // this thread's rows of the chunk: i_hi - 8 and i_hi
    uint32_t qf[8][4];
#pragma unroll
    for (int kk = 0; kk < 8; ++kk)
        if (kk < ksteps) cm_ldm4(qf[kk], cm_smem(Qs + (rw * 16 + (lane & 15)) * qs + kk * 16 + 8 * (lane >> 4)));
    float p[8][4];
#pragma unroll
    for (int nt = 0; nt < 8; ++nt) p[nt][0] = p[nt][1] = p[nt][2] = p[nt][3] = 0.f;
#pragma unroll
    for (int np = 0; np < 4; ++np) {
        if (np > rw) continue;            // keys after this warp's last row
#pragma unroll
        for (int kk = 0; kk < 8; ++kk) {
            if (kk >= ksteps) continue;
            uint32_t bf[4];
            cm_ldm4(bf, cm_smem(Ks + (np * 16 + ((lane >> 4) << 3) + (lane & 7)) * qs + kk * 16 + (((lane >> 3) & 1) << 3)));
            cm_mma(p[2 * np], qf[kk], bf[0], bf[1]);
            cm_mma(p[2 * np + 1], qf[kk], bf[2], bf[3]);
        }
    }
    const float m_before = __ldcg(work.m_before + ch);
    const float e_lo = cl[i_hi - 8] - mi[i_hi - 8], e_hi = cl[i_hi] - mi[i_hi];     // c_i - m_i
    float den_lo = 0.f, den_hi = 0.f;
#pragma unroll
    for (int nt = 0; nt < 8; ++nt) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = i_hi - 8 + 8 * (e >> 1), j = nt * 8 + 2 * tq + (e & 1);
            p[nt][e] = (j <= i && i < L) ? p[nt][e] * a.q_scale * exp2f(((e >> 1) ? e_hi : e_lo) + (ig[j] - cl[j])) : 0.f;
            if (e >> 1) den_hi += p[nt][e]; else den_lo += p[nt][e];
        }
    }
#pragma unroll
    for (int off = 1; off < 4; off <<= 1) {
        den_lo += __shfl_xor_sync(0xffffffffu, den_lo, off);
        den_hi += __shfl_xor_sync(0xffffffffu, den_hi, off);
    }
    // ---- O = P V + w_i Q S ----
    float o[4][4], o2[4][4];          // column tiles 4 cw .. 4 cw + 3 of the block
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) { o[nt][0] = o[nt][1] = o[nt][2] = o[nt][3] = 0.f; o2[nt][0] = o2[nt][1] = o2[nt][2] = o2[nt][3] = 0.f; }
#pragma unroll
    for (int kb = 0; kb < 4; ++kb) {
        if (kb > rw) continue;
        uint32_t pa[4], pb[4];
        cm_split(p[2 * kb][0], p[2 * kb][1], pa[0], pb[0]);
        cm_split(p[2 * kb][2], p[2 * kb][3], pa[1], pb[1]);
        cm_split(p[2 * kb + 1][0], p[2 * kb + 1][1], pa[2], pb[2]);
        cm_split(p[2 * kb + 1][2], p[2 * kb + 1][3], pa[3], pb[3]);
#pragma unroll
        for (int nl = 0; nl < 2; ++nl) {
            const int nb = 2 * cw + nl;
            if (2 * nb >= nt_count) continue;
            uint32_t bf[4];
            cm_ldm4t(bf, cm_smem(Vh + (kb * 16 + (((lane >> 3) & 1) << 3) + (lane & 7)) * vs + nb * 16 + ((lane >> 4) << 3)));
            cm_mma(o[2 * nl], pa, bf[0], bf[1]);
            cm_mma(o[2 * nl + 1], pa, bf[2], bf[3]);
            cm_mma(o[2 * nl], pb, bf[0], bf[1]);
            cm_mma(o[2 * nl + 1], pb, bf[2], bf[3]);
        }
    }
#pragma unroll
    for (int kk = 0; kk < 8; ++kk) {
        if (kk >= ksteps) continue;
#pragma unroll
        for (int nl = 0; nl < 2; ++nl) {
            const int nb = 2 * cw + nl;
            if (2 * nb >= nt_count) continue;
            const int off = (kk * 16 + (((lane >> 3) & 1) << 3) + (lane & 7)) * vs + nb * 16 + ((lane >> 4) << 3);
            uint32_t bh[4], bl[4];
            cm_ldm4t(bh, cm_smem(Sh + off));
            cm_ldm4t(bl, cm_smem(Sl + off));
            cm_mma(o2[2 * nl], qf[kk], bh[0], bh[1]);
            cm_mma(o2[2 * nl + 1], qf[kk], bh[2], bh[3]);
            cm_mma(o2[2 * nl], qf[kk], bl[0], bl[1]);
            cm_mma(o2[2 * nl + 1], qf[kk], bl[2], bl[3]);
        }
    }
    __syncthreads();                  // qn
    const float w_lo = a.q_scale * exp2f(e_lo + m_before), w_hi = a.q_scale * exp2f(e_hi + m_before);
    const float inv_lo = 1.0f / (fmaxf(fabsf(fmaf(w_lo, qn[i_hi - 8], den_lo)), exp2f(-mi[i_hi - 8])) + a.den_eps);
    const float inv_hi = 1.0f / (fmaxf(fabsf(fmaf(w_hi, qn[i_hi], den_hi)), exp2f(-mi[i_hi])) + a.den_eps);
    float* out_lo = a.out + (long long)(row0 + t0 + i_hi - 8) * a.n_heads * vdim + (long long)h * vdim + c0;
    float* out_hi = out_lo + 8LL * a.n_heads * vdim;
#pragma unroll
    for (int nl = 0; nl < 4; ++nl) {
        const int nt = 4 * cw + nl;
        if (nt >= nt_count) continue;
        const int c = nt * 8 + 2 * tq;
        if (i_hi - 8 < L) *reinterpret_cast<float2*>(out_lo + c) = make_float2(fmaf(w_lo, o2[nl][0], o[nl][0]) * inv_lo, fmaf(w_lo, o2[nl][1], o[nl][1]) * inv_lo);
        if (i_hi < L) *reinterpret_cast<float2*>(out_hi + c) = make_float2(fmaf(w_hi, o2[nl][2], o[nl][2]) * inv_hi, fmaf(w_hi, o2[nl][3], o[nl][3]) * inv_hi);
    }
}

// S' = 2^(c + m - m') S + 2^(A - m') U over a sequence's chunks, a thread per four elements of S; the last block of a
// (sequence, head) does the same for n, keeps m, and leaves both in every copy the scan's blocks read.
__global__ void __launch_bounds__(128) mm_scan_kernel(MatrixMemoryArgs a, ChunkWork work) {
    const int seq = blockIdx.x, h = blockIdx.y;
    const int row0 = a.seq_start[seq], n = a.seq_start[seq + 1] - row0;
    if (n <= 0 || a.tok_pos[row0] < 0) return;
    int first = 0;                                  // the step's chunks before this sequence's
    for (int s = 0; s < seq; ++s) {
        const int k = a.seq_start[s + 1] - a.seq_start[s];
        if (k > 0 && a.tok_pos[a.seq_start[s]] >= 0) first += (k + CM_CHUNK - 1) / CM_CHUNK;
    }
    const bool for_n = blockIdx.z == gridDim.z - 1;
    const long long per = for_n ? (long long)a.dim : (long long)a.dim * a.vdim;          // a multiple of 4 (both sizes are multiples of 16)
    const long long e = 4 * ((for_n ? 0LL : (long long)blockIdx.z * blockDim.x) + threadIdx.x);
    const long long head = (long long)a.slots[seq] * a.n_heads + h;
    const int copies = (a.vdim + MM_COLS - 1) / MM_COLS;
    float* N = a.norm + head * copies * (a.dim + 1);
    if (e >= per) return;
    float4 s;
    if (for_n) s = make_float4(N[e], N[e + 1], N[e + 2], N[e + 3]);
    else s = *reinterpret_cast<const float4*>(a.state + head * per + e);
    rdl_grid_wait();
    rdl_grid_launch_dependents();
    float m = __ldcg(work.m_first + (long long)seq * a.n_heads + h);
    const int chunks = (n + CM_CHUNK - 1) / CM_CHUNK;
    const long long ch0 = (long long)first * a.n_heads + h;
    float4* w = reinterpret_cast<float4*>((for_n ? work.n_work : work.s_work) + ch0 * per + e);
    const float2* tot = reinterpret_cast<const float2*>(work.totals) + ch0;
    const long long step = (long long)a.n_heads * per / 4;
    // four chunks' values are asked for while the four before them are summed and stored: loads stay in flight throughout
    float4 u[4], nx[4];
    float2 d[4], nd[4];
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        u[i] = i < chunks ? __ldcg(w + i * step) : zero;
        d[i] = i < chunks ? __ldcg(tot + (long long)i * a.n_heads) : make_float2(0.f, 0.f);
    }
    for (int c = 0; c < chunks; c += 4) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            nx[i] = c + 4 + i < chunks ? __ldcg(w + (4 + i) * step) : zero;
            nd[i] = c + 4 + i < chunks ? __ldcg(tot + (long long)(c + 4 + i) * a.n_heads) : make_float2(0.f, 0.f);
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            if (c + i < chunks) {
                __stcg(w + i * step, s);
                if (for_n && threadIdx.x == 0) work.m_before[ch0 + (long long)(c + i) * a.n_heads] = m;
                const float m_new = fmaxf(d[i].x + m, d[i].y);
                const float keep = exp2f(d[i].x + m - m_new), take = exp2f(d[i].y - m_new);
                m = m_new;
                s.x = fmaf(keep, s.x, take * u[i].x); s.y = fmaf(keep, s.y, take * u[i].y);
                s.z = fmaf(keep, s.z, take * u[i].z); s.w = fmaf(keep, s.w, take * u[i].w);
            }
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) { u[i] = nx[i]; d[i] = nd[i]; }
        w += 4 * step;
    }
    if (!for_n) {
        *reinterpret_cast<float4*>(a.state + head * per + e) = s;
        return;
    }
    for (int c = 0; c < copies; ++c) {
        float* to = N + (long long)c * (a.dim + 1);
        to[e] = s.x; to[e + 1] = s.y; to[e + 2] = s.z; to[e + 3] = s.w;
        if (threadIdx.x == 0) to[a.dim] = m;
    }
}

long long round4(long long n) { return (n + 3) / 4 * 4; }

ChunkWork work_at(float* base, long long chunks, int n_seqs, int n_heads, int dim, int vdim, long long* floats) {
    ChunkWork w;
    float* p = base;
    w.totals = p; p += round4(2 * chunks * n_heads);
    w.m_before = p; p += round4(chunks * n_heads);
    w.m_first = p; p += round4((long long)n_seqs * n_heads);
    w.n_work = p; p += chunks * n_heads * dim;
    w.s_work = p; p += chunks * n_heads * dim * vdim;
    if (floats) *floats = p - base;
    return w;
}

}  // namespace

extern "C" long long rdl_matrix_memory_chunked_work_bytes(int n_tokens, int n_seqs, int n_heads, int dim, int vdim) {
    long long floats = 0;
    work_at(nullptr, cm_max_chunks(n_tokens, n_seqs), n_seqs, n_heads, dim, vdim, &floats);
    return floats * (long long)sizeof(float);
}

extern "C" int rdl_matrix_memory_chunked(const MatrixMemoryArgs* a, void* work, long long work_bytes, void* stream) {
    if (int e = rdl_check_matrix_memory_args(a, "matrix_memory_chunked")) return e;
    RDL_REQUIRE(a->dtype == RDL_BF16, "matrix_memory_chunked: bfloat16 rows only");
    RDL_REQUIRE(a->dim % 16 == 0 && a->dim >= 16 && a->dim <= 128 && a->vdim % 16 == 0 && a->vdim >= 16,
                "matrix_memory_chunked: dim %d and vdim %d must be multiples of 16, dim at most 128", a->dim, a->vdim);
    RDL_REQUIRE(((uintptr_t)a->rows & 15) == 0 && a->row_stride % 8 == 0 && a->q_col % 8 == 0 && a->k_col % 8 == 0 && a->v_col % 8 == 0,
                "matrix_memory_chunked: rows and the columns of q, k and v must start on 16-byte boundaries");
    RDL_REQUIRE(((uintptr_t)a->out & 7) == 0 && ((uintptr_t)a->state & 15) == 0 && ((uintptr_t)work & 15) == 0,
                "matrix_memory_chunked: the output must be 8-byte aligned, state and work buffer 16-byte aligned");
    if (a->n_tokens == 0 || a->n_seqs == 0) return 0;
    RDL_REQUIRE(work && work_bytes >= rdl_matrix_memory_chunked_work_bytes(a->n_tokens, a->n_seqs, a->n_heads, a->dim, a->vdim),
                "matrix_memory_chunked: the work buffer is too small");
    const int max_chunks = cm_max_chunks(a->n_tokens, a->n_seqs);
    const ChunkWork w = work_at((float*)work, max_chunks, a->n_seqs, a->n_heads, a->dim, a->vdim, nullptr);
    const int qs = a->dim + CM_PAD, vs = MMC_COLS + CM_PAD;
    const size_t smem_u = (size_t)(CM_CHUNK * qs + 2 * CM_CHUNK * vs) * 2;
    const size_t smem_o = (size_t)(2 * CM_CHUNK * qs + CM_CHUNK * vs + 2 * a->dim * vs) * 2;
    static bool opted = false;
    if (!opted) {
        RDL_CUDA(cudaFuncSetAttribute(mm_chunk_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, 112 * 1024), "matrix_memory_chunked");
        opted = true;
    }
    cudaStream_t st = (cudaStream_t)stream;
    const dim3 grid(max_chunks, a->n_heads, (a->vdim + MMC_COLS - 1) / MMC_COLS);
    RDL_CHECK_EX(rdl_launch(mm_chunk_kernel<false>, grid, dim3(MMC_THREADS), smem_u, st, *a, w), "matrix_memory_chunked (chunk states)");
    const long long per = (long long)a->dim * a->vdim;
    RDL_CHECK_EX(rdl_launch(mm_scan_kernel, dim3(a->n_seqs, a->n_heads, (unsigned)((per / 4 + 127) / 128) + 1), dim3(128), 0, st, *a, w), "matrix_memory_chunked (scan)");
    RDL_CHECK_EX(rdl_launch(mm_chunk_kernel<true>, grid, dim3(MMC_THREADS), smem_o, st, *a, w), "matrix_memory_chunked (outputs)");
    return 0;
}
