// Latent attention on the tensor cores: BF16 cache rows, queries carried into latent space, many (token, head) rows per
// cached row. The rows of a run of n tokens are its n * heads (token, head) pairs, laid end to end and cut into tiles of
// 16 * MT rows, whatever the head count; every row carries its own causal limit. Grid (row tiles of all runs, splits of the
// visible positions); partials go where latent_attn_kernel puts them and are merged by the same kernels.
//
// A CTA holds its query tile in shared memory and streams the cache in tiles of 32 positions through a ring of cp.async
// stages, each row read once: the first `rank` elements of a row are the value, all of it is the key. GR groups of 8 warps
// share the query tile and are otherwise independent: each walks its own split of the positions with its own ring and its
// own barrier, so one group's barriers and softmax hide behind the other's products. A group of 8 warps:
//   S = Q K^T   a warp takes all rows, 16 positions and a quarter of the columns, so that shared memory is read little more
//               than once; f32 accumulation, the four partial scores meet in shared memory
//   softmax     256 / (16 MT) neighbouring threads per row; running maximum and sum in f32; the weights are split into BF16
//               high and low parts, so their products with the BF16 values lose nothing that f32 would keep
//   O += P V    every warp owns NT * 8 latent columns of all rows
#pragma once
#include "attention_mma.cuh"
#include "layered_ops.cuh"

namespace oxg4 {

constexpr int kLmThreads = 256;                      // of a group
constexpr int kLmWarps = kLmThreads / 32;
constexpr int kLmTile = 32;                          // cache positions per tile

struct LatentMmaArgs {
    // queries in f32: latent part at q_abs + row * abs_row + head * abs_head, rotated part likewise
    const float *q_abs, *q_rot;
    size_t abs_row, rot_row;
    int abs_head, rot_head;
    int heads, rank, rot;
    float scale;
    RunRows rows;
    int runs;
    int step_tiles;                      // > 0: a decode step (run r is row r, one token): row tiles per run
    RowCache cache;
    AttnPart part;
};

DEVINL void cp_async16(uint32_t dst, const void* src, bool valid) {
    const int n = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
DEVINL void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> DEVINL void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

constexpr int kLmKS = 4;                             // quarters of the columns in the score products
// A row's scores, four partial sums of 36 floats each; the row's weights (high and low BF16 parts) replace them. The stride is
// an odd number of 16-byte pieces: ldmatrix without bank conflicts.
constexpr int kLmRowBytes = 592, kLmScoreLd = 36, kLmLowBytes = 80;

// shared memory of a group besides the query tile: ring, scores / weights, rescale factors
template <int MT, int NST>
__host__ __device__ constexpr size_t latent_mma_group_bytes(int ld) {
    return (size_t)NST * kLmTile * (ld + 8) * 2 + MT * 16 * kLmRowBytes + MT * 16 * 4;
}
template <int MT, int NST, int GR>
inline size_t latent_mma_smem(int ld) {
    return (size_t)MT * 16 * (ld + 8) * 2 + GR * latent_mma_group_bytes<MT, NST>(ld) + MT * 16 * 4;
}

// NST: stages of a group's ring
template <int MT, int NT, int NST, int GR>
__global__ void __launch_bounds__(kLmThreads * GR, 1) latent_mma_kernel(const LatentMmaArgs a) {
    constexpr int ROWS = MT * 16, NB = kLmTile;
    // one row tile: the warp's query fragments stay in registers (two groups fit only for cache rows below 768 elements)
    constexpr bool QREG = MT == 1 && GR == 2;
    constexpr int QSTEPS = QREG ? 768 / 16 / kLmKS : 1;
    static_assert(kLmWarps == 2 * kLmKS && NB == 32 && NT % 2 == 0, "tile shape");
    constexpr int TPR = kLmThreads / ROWS;           // threads per row in the softmax
    constexpr int PPT = NB / TPR;                    // positions per thread
    constexpr int RPW = NB / kLmWarps;               // cache rows a warp loads per tile
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int ld = a.cache.ld, ldp = ld + 8, DK = a.rank + a.rot;
    const int grp = GR > 1 ? threadIdx.x / kLmThreads : 0, tid = threadIdx.x % kLmThreads, lane = tid & 31, warp = tid >> 5;
    uint16_t* sq = reinterpret_cast<uint16_t*>(smem_raw);            // [ROWS][ldp]
    int* s_pos = reinterpret_cast<int*>(sq + (size_t)ROWS * ldp);    // [ROWS] last visible position, -1: no row
    uint16_t* skv = reinterpret_cast<uint16_t*>(reinterpret_cast<unsigned char*>(s_pos + ROWS) + grp * latent_mma_group_bytes<MT, NST>(ld));
    unsigned char* sp = reinterpret_cast<unsigned char*>(skv + (size_t)NST * NB * ldp);   // [ROWS] rows of kLmRowBytes
    float* s_alpha = reinterpret_cast<float*>(sp + ROWS * kLmRowBytes);      // [ROWS]
    __shared__ int s_run, s_first;
    pdl_wait();
    pdl_launch();
    // the longest rows are at the end of a run: they start first
    const int t = gridDim.x - 1 - blockIdx.x;
    if (a.step_tiles == 0 && threadIdx.x < 32) {
        int run, first;
        find_row_tile(a.rows, a.runs, a.heads, ROWS, t, run, first);
        if (lane == 0) { s_run = run; s_first = first; }
    }
    int run, first, row0, n_flat;
    if (a.step_tiles > 0) {
        run = row0 = t / a.step_tiles;
        first = t % a.step_tiles * ROWS;
        n_flat = a.heads;
    } else {
        __syncthreads();
        run = s_run;
        first = s_first;
        if (run < 0) return;
        row0 = a.rows.row0[run];
        n_flat = a.rows.n[run] * a.heads;
    }
    if (a.rows.tok[row0] == kInactiveToken) return;
    const int seq = a.rows.seq_of(row0);
    const int n_here = min(ROWS, n_flat - first);
    const size_t flat0 = (size_t)row0 * a.heads + first;             // global (row, head) index of the tile's first row
    const int visible = a.rows.pos[(flat0 + n_here - 1) / a.heads] + 1;
    const int tiles = (visible + NB - 1) / NB, per = (tiles + a.part.splits - 1) / a.part.splits;
    const int split = blockIdx.y * GR + grp;
    const int tile0 = split * per, tile1 = min(tiles, tile0 + per);
    const uint16_t* pool = (const uint16_t*)a.cache.pool;
    // a lane looks up the page of one of its warp's rows, one tile ahead of the copies
    size_t row_off = 0;
    bool row_ok = false;
    auto look_up = [&](int tile) {
        const int p = tile * NB + warp * RPW + lane;
        row_ok = lane < RPW && tile < tile1 && p < visible;
        row_off = row_ok ? a.cache.row(seq, p) : 0;
    };
    const int chunks = ld / 8;
    auto load_tile = [&](int stage) {
        const unsigned valid = __ballot_sync(0xffffffffu, row_ok);
        const uint32_t dst = smem_u32(skv + ((size_t)stage * NB + warp * RPW) * ldp) + lane * 16;
#pragma unroll
        for (int i = 0; i < RPW; ++i) {
            const uint16_t* src = pool + __shfl_sync(0xffffffffu, row_off, i) + lane * 8;
            const bool ok = (valid >> i) & 1;
            const uint32_t d = dst + i * ldp * 2;
#pragma unroll
            for (int c = 0; c < 3; ++c)
                if (lane + 32 * c < chunks) cp_async16(d + c * 512, src + c * 256, ok);
            for (int c = 3; lane + 32 * c < chunks; ++c) cp_async16(d + c * 512, src + c * 256, ok);
        }
    };
    look_up(tile0);
#pragma unroll
    for (int i = 0; i < NST - 1; ++i) {
        if (tile0 + i < tile1) load_tile(i);
        cp_async_commit();                                           // one group per tile, empty past the end
        look_up(tile0 + i + 1);
    }
    if (threadIdx.x < ROWS) s_pos[threadIdx.x] = threadIdx.x < n_here ? a.rows.pos[(flat0 + threadIdx.x) / a.heads] : -1;
    for (int i = grp * kLmWarps + warp; i < ROWS; i += kLmWarps * GR) {
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
    __syncthreads();
    // ---- from here on the groups go their own ways ----
    float* part_ml = a.part.ml + 2 * ((size_t)split * a.part.rows + flat0);
    if (tile0 >= tile1) {
        if (tid < n_here) { part_ml[2 * tid] = -INFINITY; part_ml[2 * tid + 1] = 0.0f; }
        return;
    }
    auto group_sync = [&]() { asm volatile("bar.sync %0, %1;" ::"r"(1 + grp), "n"(kLmThreads) : "memory"); };
    float acc[MT][NT][4];
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int j = 0; j < NT; ++j) acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.0f;
    const int srow = tid / TPR, sub = tid % TPR;
    const float scale2 = a.scale * 1.4426950408889634f;              // scores in units of log 2
    float m_run = -INFINITY, l_run = 0.0f;                           // of row srow (the same in its TPR threads)
    const int my_pos = s_pos[srow];
    // scores of this warp: 16 positions from s_n0 on, nk steps of 16 columns from s_k0 on (ld is a multiple of 16)
    const int steps = (ld / 16 + kLmKS - 1) / kLmKS, s_kq = warp / 2, s_n0 = (warp & 1) * 16;
    const int s_k0 = min(ld, s_kq * steps * 16), nk = min(ld - s_k0, steps * 16) / 16;
    const uint32_t q_base = smem_u32(sq) + ((lane & 15) * ldp + (lane >> 4) * 8 + s_k0) * 2;
    uint32_t qf[QSTEPS][4];
    if constexpr (QREG) {
#pragma unroll
        for (int k = 0; k < QSTEPS; ++k)
            if (k < nk) ldmatrix_x4(qf[k], q_base + k * 32);
    }
    const int v_col0 = warp * NT * 8;
    int stage = 0;
    for (int tile = tile0; tile < tile1; ++tile) {
        cp_async_wait<NST - 2>();
        group_sync();                                                // tile landed; the group is done with the tile before
        {
            const int ahead = stage == 0 ? NST - 1 : stage - 1;
            if (tile + NST - 1 < tile1) load_tile(ahead);
            cp_async_commit();
            look_up(tile + NST);
        }
        const uint32_t kv = smem_u32(skv + (size_t)stage * NB * ldp);
        stage = stage + 1 == NST ? 0 : stage + 1;
        {
            float s[MT][2][4];
#pragma unroll
            for (int i = 0; i < MT; ++i)
#pragma unroll
                for (int j = 0; j < 2; ++j) s[i][j][0] = s[i][j][1] = s[i][j][2] = s[i][j][3] = 0.0f;
            const uint32_t kb = kv + ((s_n0 + (lane >> 4) * 8 + (lane & 7)) * ldp + ((lane >> 3) & 1) * 8 + s_k0) * 2;
            if constexpr (QREG) {
#pragma unroll
                for (int k = 0; k < QSTEPS; ++k)
                    if (k < nk) {
                        uint32_t b[4];
                        ldmatrix_x4(b, kb + k * 32);
                        mma_bf16_16816(s[0][0], qf[k], b[0], b[1]);
                        mma_bf16_16816(s[0][1], qf[k], b[2], b[3]);
                    }
            } else {
#pragma unroll 3
                for (int k = 0; k < nk; ++k) {
                    uint32_t b[4], q[MT][4];
                    ldmatrix_x4(b, kb + k * 32);
#pragma unroll
                    for (int i = 0; i < MT; ++i) ldmatrix_x4(q[i], q_base + i * 16 * ldp * 2 + k * 32);
#pragma unroll
                    for (int i = 0; i < MT; ++i) {
                        mma_bf16_16816(s[i][0], q[i], b[0], b[1]);
                        mma_bf16_16816(s[i][1], q[i], b[2], b[3]);
                    }
                }
            }
#pragma unroll
            for (int i = 0; i < MT; ++i)
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    float* dst = reinterpret_cast<float*>(sp + (i * 16 + (lane >> 2)) * kLmRowBytes) + s_kq * kLmScoreLd + s_n0 + j * 8 + (lane & 3) * 2;
                    *reinterpret_cast<float2*>(dst) = make_float2(s[i][j][0], s[i][j][1]);
                    *reinterpret_cast<float2*>(dst + 8 * kLmRowBytes / 4) = make_float2(s[i][j][2], s[i][j][3]);
                }
        }
        group_sync();
        {
            const int lim = my_pos - tile * NB;                      // last visible column of this row
            float v[PPT], mx = -INFINITY;
#pragma unroll
            for (int j = 0; j < PPT; j += 2) {                       // pairs of neighbouring positions
                const int c = 2 * sub + j * TPR;
                const float* src = reinterpret_cast<const float*>(sp + srow * kLmRowBytes) + c;
                float2 x = *reinterpret_cast<const float2*>(src);
#pragma unroll
                for (int q = 1; q < kLmKS; ++q) {
                    const float2 y = *reinterpret_cast<const float2*>(src + q * kLmScoreLd);
                    x.x += y.x;
                    x.y += y.y;
                }
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
            __syncwarp();                                            // a row's threads are one warp's: its scores are all read
#pragma unroll
            for (int j = 0; j < PPT; j += 2) {
                const float e0 = exp2f(v[j] - base), e1 = exp2f(v[j + 1] - base);
                sum += e0 + e1;
                uint32_t hi, lo;
                split_pack(e0, e1, hi, lo);
                const int c = 2 * sub + j * TPR;
                *reinterpret_cast<uint32_t*>(sp + srow * kLmRowBytes + c * 2) = hi;
                *reinterpret_cast<uint32_t*>(sp + srow * kLmRowBytes + kLmLowBytes + c * 2) = lo;
            }
            l_run = l_run * alpha + sum;                             // this thread's positions only; added up at the end
            m_run = m_new;
            if (sub == 0) s_alpha[srow] = alpha;
        }
        group_sync();
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
            const uint32_t p_base = smem_u32(sp) + (lane & 15) * kLmRowBytes + (lane >> 4) * 16;
            const uint32_t v_base = kv + ((lane & 15) * ldp + v_col0 + (lane >> 4) * 8) * 2;
#pragma unroll
            for (int k = 0; k < NB; k += 16) {
                uint32_t ph[MT][4], pl[MT][4];
#pragma unroll
                for (int i = 0; i < MT; ++i) {
                    ldmatrix_x4(ph[i], p_base + i * 16 * kLmRowBytes + k * 2);
                    ldmatrix_x4(pl[i], p_base + i * 16 * kLmRowBytes + kLmLowBytes + k * 2);
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
                        }
#pragma unroll
                        for (int i = 0; i < MT; ++i) {
                            mma_bf16_16816(acc[i][j], pl[i], b[0], b[1]);
                            mma_bf16_16816(acc[i][j + 1], pl[i], b[2], b[3]);
                        }
                    }
                }
            }
        }
    }
#pragma unroll
    for (int o = TPR / 2; o > 0; o >>= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, o);
    if (sub == 0 && srow < n_here) { part_ml[2 * srow] = m_run * 0.6931471805599453f; part_ml[2 * srow + 1] = l_run; }
    float* po = a.part.o + ((size_t)split * a.part.rows + flat0) * a.rank;
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
