// Latent attention on the tensor cores: BF16 cache rows, queries carried into latent space, many (token, head) rows per
// cached row. The rows of a run of n tokens are its n * heads (token, head) pairs, laid end to end and cut into tiles of
// 16 * MT rows, whatever the head count; every row carries its own causal limit. Grid (row tiles of all runs, splits of the
// visible positions); partials go where latent_attn_kernel puts them and are merged by the same kernels.
//
// A CTA holds its query tile in shared memory and streams the cache in tiles of NB positions, two stages of
// cp.async, each row read once: the first `rank` elements of a row are the value, all of it is the key. 8 warps:
//   S = Q K^T   16 x 8 tiles of the score block dealt to the warps, f32 accumulation, scaled and masked into shared memory
//   softmax     256 / (16 MT) neighbouring threads per row; running maximum and sum in f32; the weights are split into BF16
//               high and low parts, so their products with the BF16 values lose nothing that f32 would keep
//   O += P V    every warp owns NT * 8 latent columns of all rows
#pragma once
#include "attention_mma.cuh"
#include "layered_ops.cuh"

namespace oxg4 {

constexpr int kLmThreads = 256;
constexpr int kLmWarps = kLmThreads / 32;

struct LatentMmaArgs {
    // queries in f32: latent part at q_abs + row * abs_row + head * abs_head, rotated part likewise
    const float *q_abs, *q_rot;
    size_t abs_row, rot_row;
    int abs_head, rot_head;
    int heads, rank, rot;
    float scale;
    RunRows rows;
    int runs;
    LatentCache cache;
    LatentPart part;
};

DEVINL void cp_async16(uint32_t dst, const void* src, bool valid) {
    const int n = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
DEVINL void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> DEVINL void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

template <int MT, int NB>
inline size_t latent_mma_smem(int ld) {
    const size_t rows = MT * 16, ldp = ld + 8;
    return (rows + 2 * NB) * ldp * 2 + 2 * rows * (NB + 8) * 2 + rows * (NB + 4) * 4 + 3 * rows * 4 + 64;
}

// KQ > 0: the query fragments of a warp's score tile stay in registers (KQ steps of 16 columns, rows of at most 16 KQ
// elements), which leaves shared memory to the cache rows.
template <int MT, int NT, int NB, int KQ>
__global__ void __launch_bounds__(kLmThreads, 1) latent_mma_kernel(const LatentMmaArgs a) {
    constexpr int ROWS = MT * 16;
    constexpr int SN = NB / 8;                       // score columns in MMA tiles
    constexpr int SPW = MT * SN / kLmWarps;          // score tiles per warp
    static_assert(MT * SN % kLmWarps == 0 && NT % 2 == 0 && NB % (2 * kLmThreads / ROWS) == 0, "tile shape");
    constexpr int TPR = kLmThreads / ROWS;           // threads per row in the softmax
    constexpr int PPT = NB / TPR;                    // positions per thread
    constexpr int PLD = NB + 8, SLD = NB + 4;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int ld = a.cache.ld, ldp = ld + 8, DK = a.rank + a.rot;
    uint16_t* sq = reinterpret_cast<uint16_t*>(smem_raw);            // [ROWS][ldp]
    uint16_t* skv = sq + (size_t)ROWS * ldp;                         // [2][NB][ldp]
    uint16_t* sp = skv + (size_t)2 * NB * ldp;                       // [2 (hi, lo)][ROWS][PLD]
    float* ss = reinterpret_cast<float*>(sp + 2 * ROWS * PLD);       // [ROWS][SLD]
    float* s_alpha = ss + ROWS * SLD;                                // [ROWS]
    int* s_pos = reinterpret_cast<int*>(s_alpha + ROWS);             // [ROWS] last visible position, -1: no row
    __shared__ int s_run, s_first;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    pdl_wait();
    pdl_launch();
    // the longest rows are at the end of a run: they start first
    const int t = gridDim.x - 1 - blockIdx.x;
    if (warp == 0) {
        int base = 0, run = -1, first = 0;
        for (int r0 = 0; r0 < a.runs && run < 0; r0 += 32) {
            const int r = r0 + lane;
            const int nt = r < a.runs ? (a.rows.n[r] * a.heads + ROWS - 1) / ROWS : 0;
            int inc = nt;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int v = __shfl_up_sync(0xffffffffu, inc, o);
                if (lane >= o) inc += v;
            }
            const int lo = base + inc - nt;
            const unsigned hit = __ballot_sync(0xffffffffu, t >= lo && t < lo + nt);
            if (hit) {
                const int src = __ffs(hit) - 1;
                run = r0 + src;
                first = (t - __shfl_sync(0xffffffffu, lo, src)) * ROWS;
            }
            base += __shfl_sync(0xffffffffu, inc, 31);
        }
        if (lane == 0) { s_run = run; s_first = first; }
    }
    __syncthreads();
    const int run = s_run, first = s_first;
    if (run < 0) return;
    const int row0 = a.rows.row0[run], n_flat = a.rows.n[run] * a.heads;
    if (a.rows.tok[row0] == kInactiveToken) return;
    const int seq = a.rows.seq_of(row0);
    const int n_here = min(ROWS, n_flat - first);
    const size_t flat0 = (size_t)row0 * a.heads + first;             // global (row, head) index of the tile's first row
    if (tid < ROWS) s_pos[tid] = tid < n_here ? a.rows.pos[(flat0 + tid) / a.heads] : -1;
    const int visible = a.rows.pos[(flat0 + n_here - 1) / a.heads] + 1;
    const int tiles = (visible + NB - 1) / NB, per = (tiles + a.part.splits - 1) / a.part.splits;
    const int tile0 = blockIdx.y * per, tile1 = min(tiles, tile0 + per);
    float* part_ml = a.part.ml + 2 * ((size_t)blockIdx.y * a.part.rows + flat0);
    if (tile0 >= tile1) {
        if (tid < n_here) { part_ml[2 * tid] = -INFINITY; part_ml[2 * tid + 1] = 0.0f; }
        return;
    }
    const uint16_t* pool = (const uint16_t*)a.cache.pool;
    auto load_tile = [&](int tile, int stage) {
        constexpr int RPW = NB / kLmWarps;                           // rows per warp; one lane looks up each row's page
        const int chunks = ld / 8, p = tile * NB + warp * RPW + lane;
        const bool mine = lane < RPW && p < visible;
        const size_t off = mine ? a.cache.row(seq, p) : 0;
        const unsigned valid = __ballot_sync(0xffffffffu, mine);
        const uint32_t dst = smem_u32(skv + ((size_t)stage * NB + warp * RPW) * ldp);
#pragma unroll
        for (int i = 0; i < RPW; ++i) {
            const uint16_t* src = pool + __shfl_sync(0xffffffffu, off, i) + lane * 8;
            const bool ok = (valid >> i) & 1;
            const uint32_t d = dst + i * ldp * 2 + lane * 16;
#pragma unroll
            for (int c = 0; c < 3; ++c)                              // cache rows of up to 768 elements
                if (lane + 32 * c < chunks) cp_async16(d + c * 512, src + c * 256, ok);
            for (int c = 3; lane + 32 * c < chunks; ++c) cp_async16(d + c * 512, src + c * 256, ok);
        }
    };
    load_tile(tile0, 0);
    cp_async_commit();
    for (int i = warp; i < ROWS; i += kLmWarps) {
        const size_t f = flat0 + i;
        const size_t row = f / a.heads;
        const int hd = (int)(f - row * a.heads);
        const float* qa = a.q_abs + row * a.abs_row + (size_t)hd * a.abs_head;
        const float* qr = a.q_rot + row * a.rot_row + (size_t)hd * a.rot_head - a.rank;
        for (int j0 = 0; j0 < ld; j0 += 256) {
            float v[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                const int j = j0 + lane + 32 * e;
                v[e] = i < n_here && j < DK ? (j < a.rank ? qa[j] : qr[j]) : 0.0f;
            }
#pragma unroll
            for (int e = 0; e < 8; ++e)
                if (j0 + lane + 32 * e < ld) sq[(size_t)i * ldp + j0 + lane + 32 * e] = (uint16_t)f32_to_bf16_bits(v[e]);
        }
    }
    float acc[MT][NT][4];
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int j = 0; j < NT; ++j) acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.0f;
    const int srow = tid / TPR, sub = tid % TPR;
    const float scale2 = a.scale * 1.4426950408889634f;              // scores in units of log 2
    float m_run = -INFINITY, l_run = 0.0f;                           // of row srow (the same in its TPR threads)
    // score tiles of this warp: one row tile, SPW neighbouring column tiles
    const int s_mi = warp % MT, s_n0 = (warp / MT) * SPW;
    const uint32_t q_base = smem_u32(sq) + ((s_mi * 16 + (lane & 15)) * ldp + (lane >> 4) * 8) * 2;
    const int v_col0 = warp * NT * 8;
    uint32_t qf[KQ > 0 ? KQ : 1][4];
    for (int tile = tile0; tile < tile1; ++tile) {
        const int stage = (tile - tile0) & 1;
        cp_async_wait<0>();
        __syncthreads();                                             // tile landed; everyone is done with the other stage
        if (tile + 1 < tile1) {
            load_tile(tile + 1, stage ^ 1);
            cp_async_commit();
        }
        const uint32_t kv = smem_u32(skv + (size_t)stage * NB * ldp);
        {
            float s[SPW][4];
#pragma unroll
            for (int j = 0; j < SPW; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.0f;
            if constexpr (KQ > 0) {
                if (tile == tile0) {
#pragma unroll
                    for (int k = 0; k < KQ; ++k)
                        if (k * 16 < ld) ldmatrix_x4(qf[k], q_base + k * 32);
                }
                float s2[SPW][4];
#pragma unroll
                for (int j = 0; j < SPW; ++j) s2[j][0] = s2[j][1] = s2[j][2] = s2[j][3] = 0.0f;
                if constexpr (SPW == 1) {
                    // one column tile: a load brings its 8 positions for two k-steps
                    float s3[4] = {0.0f, 0.0f, 0.0f, 0.0f}, s4[4] = {0.0f, 0.0f, 0.0f, 0.0f};
                    const uint32_t kb = kv + ((s_n0 * 8 + (lane & 7)) * ldp + (lane >> 3) * 8) * 2;
#pragma unroll
                    for (int k = 0; k < KQ; k += 2) {
                        uint32_t b[4];
                        if (k * 16 + 32 <= ld) {
                            ldmatrix_x4(b, kb + k * 32);
                            mma_bf16_16816((k & 2) ? s3 : s[0], qf[k], b[0], b[1]);
                            mma_bf16_16816((k & 2) ? s4 : s2[0], qf[k + 1], b[2], b[3]);
                        } else if (k * 16 < ld) {                    // ld is a multiple of 16
                            ldmatrix_x4(b, kv + ((s_n0 * 8 + (lane & 7)) * ldp + ((lane >> 3) & 1) * 8 + k * 16) * 2);
                            mma_bf16_16816(s[0], qf[k], b[0], b[1]);
                        }
                    }
#pragma unroll
                    for (int q = 0; q < 4; ++q) s[0][q] += s3[q] + s4[q];
                } else {
                    // a pair of column tiles: a load brings 16 positions for one k-step
                    static_assert(SPW <= 2, "score tiles per warp");
                    const uint32_t kb = kv + ((s_n0 * 8 + (lane >> 4) * 8 + (lane & 7)) * ldp + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll
                    for (int k = 0; k < KQ; ++k)
                        if (k * 16 < ld) {
                            uint32_t b[4];
                            ldmatrix_x4(b, kb + k * 32);
                            mma_bf16_16816((k & 1) ? s2[0] : s[0], qf[k], b[0], b[1]);
                            mma_bf16_16816((k & 1) ? s2[1] : s[1], qf[k], b[2], b[3]);
                        }
                }
#pragma unroll
                for (int j = 0; j < SPW; ++j)
#pragma unroll
                    for (int q = 0; q < 4; ++q) s[j][q] += s2[j][q];
            } else if constexpr (SPW == 1) {
                // one column tile: a load brings its 8 positions for two k-steps
                const uint32_t kb = kv + ((s_n0 * 8 + (lane & 7)) * ldp + (lane >> 3) * 8) * 2;
                float s2[4] = {0.0f, 0.0f, 0.0f, 0.0f};
                int k = 0;
#pragma unroll 2
                for (; k + 32 <= ld; k += 32) {
                    uint32_t q0[4], q1[4], b[4];
                    ldmatrix_x4(b, kb + k * 2);
                    ldmatrix_x4(q0, q_base + k * 2);
                    ldmatrix_x4(q1, q_base + k * 2 + 32);
                    mma_bf16_16816(s[0], q0, b[0], b[1]);
                    mma_bf16_16816(s2, q1, b[2], b[3]);
                }
                if (k < ld) {                                        // ld is a multiple of 16
                    uint32_t q0[4], b[4];
                    // the upper half of the lanes addresses the same columns again: no read behind the row
                    ldmatrix_x4(b, kv + ((s_n0 * 8 + (lane & 7)) * ldp + ((lane >> 3) & 1) * 8 + k) * 2);
                    ldmatrix_x4(q0, q_base + k * 2);
                    mma_bf16_16816(s[0], q0, b[0], b[1]);
                }
#pragma unroll
                for (int q = 0; q < 4; ++q) s[0][q] += s2[q];
            } else {
                // pairs of column tiles: a load brings 16 positions for one k-step
                uint32_t kb[SPW / 2];
#pragma unroll
                for (int j = 0; j < SPW / 2; ++j)
                    kb[j] = kv + ((s_n0 * 8 + j * 16 + (lane >> 4) * 8 + (lane & 7)) * ldp + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll 4
                for (int k = 0; k < ld; k += 16) {
                    uint32_t q0[4];
                    ldmatrix_x4(q0, q_base + k * 2);
#pragma unroll
                    for (int j = 0; j < SPW / 2; ++j) {
                        uint32_t b[4];
                        ldmatrix_x4(b, kb[j] + k * 2);
                        mma_bf16_16816(s[2 * j], q0, b[0], b[1]);
                        mma_bf16_16816(s[2 * j + 1], q0, b[2], b[3]);
                    }
                }
            }
            const int r0 = s_mi * 16 + (lane >> 2);
#pragma unroll
            for (int j = 0; j < SPW; ++j) {
                const int c = (s_n0 + j) * 8 + (lane & 3) * 2;
                *reinterpret_cast<float2*>(ss + r0 * SLD + c) = make_float2(s[j][0], s[j][1]);
                *reinterpret_cast<float2*>(ss + (r0 + 8) * SLD + c) = make_float2(s[j][2], s[j][3]);
            }
        }
        __syncthreads();
        {
            const int lim = s_pos[srow] - tile * NB;                 // last visible column of this row
            float v[PPT], mx = -INFINITY;
#pragma unroll
            for (int j = 0; j < PPT; j += 2) {                       // pairs of neighbouring positions
                const int c = 2 * sub + j * TPR;
                const float2 x = *reinterpret_cast<const float2*>(ss + srow * SLD + c);
                v[j] = c <= lim ? x.x * scale2 : -INFINITY;
                v[j + 1] = c + 1 <= lim ? x.y * scale2 : -INFINITY;
                mx = fmaxf(mx, fmaxf(v[j], v[j + 1]));
            }
#pragma unroll
            for (int o = TPR / 2; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float m_new = fmaxf(m_run, mx);
            const float base = m_new == -INFINITY ? 0.0f : m_new;    // a row without a visible position so far
            const float alpha = m_new == m_run ? 1.0f : exp2f(m_run - base);
            float sum = 0.0f;
#pragma unroll
            for (int j = 0; j < PPT; j += 2) {
                const float e0 = exp2f(v[j] - base), e1 = exp2f(v[j + 1] - base);
                sum += e0 + e1;
                uint32_t hi, lo;
                split_pack(e0, e1, hi, lo);
                const int c = 2 * sub + j * TPR;
                *reinterpret_cast<uint32_t*>(sp + srow * PLD + c) = hi;
                *reinterpret_cast<uint32_t*>(sp + (ROWS + srow) * PLD + c) = lo;
            }
#pragma unroll
            for (int o = TPR / 2; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            l_run = l_run * alpha + sum;
            m_run = m_new;
            if (sub == 0) s_alpha[srow] = alpha;
        }
        __syncthreads();
        if (v_col0 < a.rank) {
            bool moved = false;
            float al[MT][2];
#pragma unroll
            for (int i = 0; i < MT; ++i) {
                al[i][0] = s_alpha[i * 16 + (lane >> 2)];
                al[i][1] = s_alpha[i * 16 + 8 + (lane >> 2)];
                moved |= al[i][0] != 1.0f || al[i][1] != 1.0f;
            }
            if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
                for (int i = 0; i < MT; ++i)
#pragma unroll
                    for (int j = 0; j < NT; ++j) {
                        acc[i][j][0] *= al[i][0]; acc[i][j][1] *= al[i][0];
                        acc[i][j][2] *= al[i][1]; acc[i][j][3] *= al[i][1];
                    }
            }
            const uint32_t p_base = smem_u32(sp) + ((lane & 15) * PLD + (lane >> 4) * 8) * 2;
            const uint32_t v_base = kv + ((lane & 15) * ldp + v_col0 + (lane >> 4) * 8) * 2;
#pragma unroll
            for (int k = 0; k < NB; k += 16) {
                uint32_t ph[MT][4], pl[MT][4];
#pragma unroll
                for (int i = 0; i < MT; ++i) {
                    ldmatrix_x4(ph[i], p_base + (i * 16 * PLD + k) * 2);
                    ldmatrix_x4(pl[i], p_base + ((ROWS + i * 16) * PLD + k) * 2);
                }
#pragma unroll
                for (int j = 0; j < NT; j += 2) {
                    if (v_col0 + j * 8 < ld) {
                        uint32_t b[4];
                        ldmatrix_x4_trans(b, v_base + (k * ldp + j * 8) * 2);
#pragma unroll
                        for (int i = 0; i < MT; ++i) {
                            mma_bf16_16816(acc[i][j], ph[i], b[0], b[1]);
                            mma_bf16_16816(acc[i][j + 1], ph[i], b[2], b[3]);
                            mma_bf16_16816(acc[i][j], pl[i], b[0], b[1]);
                            mma_bf16_16816(acc[i][j + 1], pl[i], b[2], b[3]);
                        }
                    }
                }
            }
        }
    }
    if (sub == 0 && srow < n_here) { part_ml[2 * srow] = m_run * 0.6931471805599453f; part_ml[2 * srow + 1] = l_run; }
    float* po = a.part.o + ((size_t)blockIdx.y * a.part.rows + flat0) * a.rank;
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            const int r = i * 16 + h * 8 + (lane >> 2);
            if (r >= n_here) continue;
#pragma unroll
            for (int j = 0; j < NT; ++j) {
                const int c = v_col0 + j * 8 + (lane & 3) * 2;
                float* o = po + (size_t)r * a.rank + c;
                if (c < a.rank) o[0] = acc[i][j][2 * h];
                if (c + 1 < a.rank) o[1] = acc[i][j][2 * h + 1];
            }
        }
}

}  // namespace oxg4
