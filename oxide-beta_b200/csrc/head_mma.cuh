// Grouped-query attention on the tensor cores over a paged cache of [key | value] rows: BF16 cache and queries, any key and
// value size up to 256, any number of query heads per kv head. The rows of a run of n tokens are, per kv head, its
// n * group (token, head) pairs, laid end to end and cut into tiles; every row carries its own causal limit. Grid (row tiles
// of all runs, kv heads, splits of the visible positions); the partials are merged by head_merge_kernel.
//
// A CTA streams its positions in tiles of 64 through a ring of cp.async stages: one contiguous piece of memory per cached
// token holds its key and its value. Four warps either own 16 rows each (WR = 4: prompts, many rows share a tile) or share
// 16 rows and own 16 positions of every tile each (WP = 4: decode steps, whose time is the stream of the cache). Scores,
// softmax and value product of a warp's rows and positions stay in its registers; the only barrier of a tile is the one that
// hands over the stage. Scores and running maximum and sum are f32; the weights enter the value product as BF16 high and
// low parts, so their products with the BF16 values lose nothing that f32 would keep.
#pragma once
#include "latent_mma.cuh"

namespace oxg4 {

constexpr int kHmTile = 64;                          // cache positions per tile
constexpr int kHmWarps = 4;
constexpr int kHmThreads = 32 * kHmWarps;

struct HeadMmaArgs {
    const uint16_t* q;                   // [R, heads, kd] BF16
    int heads, group, kd, vd, vdim;      // kd, vd: padded to multiples of 16; cache row = kd + vd
    float scale;
    RunRows rows;
    int runs;
    int step_tiles;                      // > 0: a decode step (run r is row r, one token): row tiles per run
    RowCache cache;
    AttnPart part;
};

// stages of the ring: as many as leave room for two CTAs on an SM (up to 128 columns)
__host__ __device__ constexpr int head_mma_stages(int cols, int wr) { return cols > 128 || (cols > 64 && wr > 1) ? 2 : 3; }
inline size_t head_mma_smem(int cols, int wr, int ld, int kd, int vd) {
    const size_t ring = (size_t)head_mma_stages(cols, wr) * kHmTile * (ld + 8) * 2;
    const size_t merge = wr == 1 ? (size_t)kHmWarps * 16 * (vd + 4) * 4 : 0;
    return (ring > merge ? ring : merge) + (size_t)wr * 16 * (kd + 8) * 2;
}

// COLS: bound on kd and vd
template <int COLS, int WR>
__global__ void __launch_bounds__(kHmThreads) head_mma_kernel(const HeadMmaArgs a) {
    constexpr int WP = kHmWarps / WR, ROWS = WR * 16, NST = head_mma_stages(COLS, WR);
    constexpr int PW = kHmTile / WP;                 // positions of a tile that are this warp's
    constexpr int KSTEPS = COLS / 16, VT = COLS / 8, ST = PW / 8;
    constexpr bool QREG = COLS <= 128;               // query fragments stay in registers
    constexpr int RPW = kHmTile / kHmWarps;          // cache rows a warp loads per tile
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int ld = a.cache.ld, ldp = ld + 8, qld = a.kd + 8;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, wr = WR > 1 ? warp : 0, wp = WR > 1 ? 0 : warp;
    uint16_t* sq = reinterpret_cast<uint16_t*>(smem_raw);            // [ROWS][qld]
    uint16_t* skv = sq + (size_t)ROWS * qld;                         // [NST][tile][ldp]
    __shared__ int s_run, s_first;
    __shared__ float s_ml[kHmWarps][16][2];
    // Rows, positions and pages were there before the preceding kernel started, and so were the cached tokens of earlier steps:
    // they are read ahead of the dependency wait. The queries and this pass's own cache rows are not.
    const int kvh = blockIdx.y, split = blockIdx.z;
    const int t = gridDim.x - 1 - blockIdx.x;        // the longest rows are at the end of a run: they start first
    int run, first, row0, n_flat;
    if (a.step_tiles > 0) {
        run = row0 = t / a.step_tiles;
        first = t % a.step_tiles * ROWS;
        n_flat = a.group;
    } else {
        if (warp == 0) {
            find_row_tile(a.rows, a.runs, a.group, ROWS, t, run, first);
            if (lane == 0) { s_run = run; s_first = first; }
        }
        __syncthreads();
        run = s_run;
        first = s_first;
        if (run < 0) {
            pdl_wait();
            pdl_launch();
            return;
        }
        row0 = a.rows.row0[run];
        n_flat = a.rows.n[run] * a.group;
    }
    if (a.rows.tok[row0] == kInactiveToken) {
        pdl_wait();
        pdl_launch();
        return;
    }
    const int seq = a.rows.seq_of(row0), n_here = min(ROWS, n_flat - first);
    const int visible = a.rows.pos[row0 + (first + n_here - 1) / a.group] + 1;
    const int tiles = (visible + kHmTile - 1) / kHmTile, per = (tiles + a.part.splits - 1) / a.part.splits;
    const int tile0 = split * per, tile1 = min(tiles, tile0 + per);
    auto part_row = [&](int i) {                     // partial of row i of this tile
        const int f = first + i;
        return (size_t)split * a.part.rows + (size_t)(row0 + f / a.group) * a.heads + kvh * a.group + f % a.group;
    };
    if (tile0 >= tile1) {
        pdl_wait();
        pdl_launch();
        if (tid < n_here) {
            float* ml = a.part.ml + 2 * part_row(tid);
            ml[0] = -INFINITY;
            ml[1] = 0.0f;
        }
        return;
    }
    const uint16_t* pool = (const uint16_t*)a.cache.pool;
    // a lane looks up the page of one of its warp's rows, one tile ahead of the copies; its place in the pages moves on tile by tile
    const int32_t* pages = a.cache.page_table + (size_t)seq * a.cache.pages_per_seq;
    const int my_row = warp * RPW + (lane & (RPW - 1));
    int page_i = (tile0 * kHmTile + my_row) / a.cache.page_tokens, page_o = (tile0 * kHmTile + my_row) % a.cache.page_tokens;
    size_t row_off = 0;
    bool row_ok = false;
    auto look_up = [&](int tile) {                   // called for tile0, tile0 + 1, ...
        row_ok = tile < tile1 && tile * kHmTile + my_row < visible;
        row_off = row_ok ? (((size_t)pages[page_i] * a.cache.kv_heads + kvh) * a.cache.page_tokens + page_o) * ld : 0;
        page_o += kHmTile;
        while (page_o >= a.cache.page_tokens) {
            page_o -= a.cache.page_tokens;
            ++page_i;
        }
    };
    constexpr int LPR = COLS >= 128 ? 32 : COLS / 4, RPI = 32 / LPR, CPL = (COLS / 4 + 31) / 32;     // lanes per row, rows at a time, pieces per lane
    const int chunk0 = lane & (LPR - 1), chunks = ld / 8;
    auto load_tile = [&](int stage) {
        const unsigned valid = __ballot_sync(0xffffffffu, row_ok);
        const uint32_t dst = smem_u32(skv + ((size_t)stage * kHmTile + warp * RPW) * ldp) + chunk0 * 16;
#pragma unroll
        for (int i = 0; i < RPW; i += RPI) {
            const int r = i + lane / LPR;
            const uint16_t* src = pool + __shfl_sync(0xffffffffu, row_off, r) + chunk0 * 8;
#pragma unroll
            for (int c = 0; c < CPL; ++c)
                if (chunk0 + 32 * c < chunks) cp_async16(dst + r * ldp * 2 + c * 512, src + c * 256, (valid >> r) & 1);
        }
    };
    const bool early = (tile0 + NST - 1) * kHmTile <= a.rows.pos[row0];      // the first tiles hold no token of this pass
    if (!early) pdl_wait();
    look_up(tile0);
#pragma unroll
    for (int i = 0; i < NST - 1; ++i) {
        if (tile0 + i < tile1) load_tile(i);
        cp_async_commit();                           // one group per tile, empty past the end
        look_up(tile0 + i + 1);
    }
    if (early) pdl_wait();
    pdl_launch();
    for (int i = tid; i < ROWS * (a.kd / 8); i += kHmThreads) {
        const int row = i / (a.kd / 8), ch = i % (a.kd / 8), f = first + row;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (row < n_here)
            v = *reinterpret_cast<const uint4*>(a.q + ((size_t)(row0 + f / a.group) * a.heads + kvh * a.group + f % a.group) * a.kd + ch * 8);
        *reinterpret_cast<uint4*>(sq + (size_t)row * qld + ch * 8) = v;
    }
    // last visible position of the two rows of this lane, -1: no row
    int lim[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        const int i = wr * 16 + h * 8 + (lane >> 2);
        lim[h] = i < n_here ? a.rows.pos[row0 + (first + i) / a.group] : -1;
    }
    __syncthreads();
    // Steps past kd multiply zero queries with columns that are there, value columns past vd are computed and not stored:
    // the loops have no branches, so the loads of a step overlap the products of the one before.
    const int ksteps = a.kd / 16, vpairs = a.vd / 16;
    const uint32_t q_base = smem_u32(sq) + ((wr * 16 + (lane & 15)) * qld + (lane >> 4) * 8) * 2;
    uint32_t qf[QREG ? KSTEPS : 1][4];
    if constexpr (QREG) {
#pragma unroll
        for (int k = 0; k < KSTEPS; ++k) {
            ldmatrix_x4(qf[k], q_base + min(k, ksteps - 1) * 32);
#pragma unroll
            for (int e = 0; e < 4; ++e) qf[k][e] = k < ksteps ? qf[k][e] : 0u;
        }
    }
    float o[VT][4];
#pragma unroll
    for (int j = 0; j < VT; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.0f;
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.0f, 0.0f};
    const float scale2 = a.scale * 1.4426950408889634f;              // scores in units of log 2
    int stage = 0;
    for (int tile = tile0; tile < tile1; ++tile) {
        cp_async_wait<NST - 2>();
        __syncthreads();                             // tile landed; every warp is done with the tile before
        {
            const int ahead = stage == 0 ? NST - 1 : stage - 1;
            if (tile + NST - 1 < tile1) load_tile(ahead);
            cp_async_commit();
            look_up(tile + NST);
        }
        const uint32_t kv = smem_u32(skv + ((size_t)stage * kHmTile + wp * PW) * ldp);
        stage = stage + 1 == NST ? 0 : stage + 1;
        // ---- scores ----
        float s[ST][4];
#pragma unroll
        for (int j = 0; j < ST; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.0f;
        const uint32_t kb = kv + (((lane >> 4) * 8 + (lane & 7)) * ldp + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll
        for (int k = 0; k < KSTEPS; ++k) {
            const int col = min(k, ksteps - 1) * 16;
            uint32_t q[4];
            if constexpr (QREG) {
#pragma unroll
                for (int e = 0; e < 4; ++e) q[e] = qf[k][e];
            } else {
                ldmatrix_x4(q, q_base + col * 2);
#pragma unroll
                for (int e = 0; e < 4; ++e) q[e] = k < ksteps ? q[e] : 0u;
            }
#pragma unroll
            for (int j = 0; j < ST; j += 2) {
                uint32_t b[4];
                ldmatrix_x4(b, kb + (j * 8 * ldp + col) * 2);
                mma_bf16_16816(s[j], q, b[0], b[1]);
                mma_bf16_16816(s[j + 1], q, b[2], b[3]);
            }
        }
        // ---- softmax: a row's scores are in the four lanes of a quad ----
        const int p0 = tile * kHmTile + wp * PW + (lane & 3) * 2;
        float alpha[2];
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            float mx = -INFINITY;
#pragma unroll
            for (int j = 0; j < ST; ++j)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    float& x = s[j][2 * h + e];
                    x = p0 + j * 8 + e <= lim[h] ? x * scale2 : -INFINITY;
                    mx = fmaxf(mx, x);
                }
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
            const float m_new = fmaxf(m_run[h], mx), base = m_new == -INFINITY ? 0.0f : m_new;
            alpha[h] = m_new == m_run[h] ? 1.0f : exp2f(m_run[h] - base);
            m_run[h] = m_new;
            float sum = 0.0f;
#pragma unroll
            for (int j = 0; j < ST; ++j)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    float& x = s[j][2 * h + e];
                    x = exp2f(x - base);
                    sum += x;
                }
            l_run[h] = l_run[h] * alpha[h] + sum;    // this lane's positions only; added up at the end
        }
        if (__any_sync(0xffffffffu, alpha[0] != 1.0f || alpha[1] != 1.0f)) {
#pragma unroll
            for (int j = 0; j < VT; ++j) {
                o[j][0] *= alpha[0]; o[j][1] *= alpha[0];
                o[j][2] *= alpha[1]; o[j][3] *= alpha[1];
            }
        }
        // ---- value product: the score registers are the operand's layout ----
        const uint32_t v_base = kv + ((lane & 15) * ldp + a.kd + (lane >> 4) * 8) * 2;
#pragma unroll
        for (int k = 0; k < PW / 16; ++k) {
            uint32_t ph[4], pl[4];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                split_pack(s[2 * k + e][0], s[2 * k + e][1], ph[2 * e], pl[2 * e]);
                split_pack(s[2 * k + e][2], s[2 * k + e][3], ph[2 * e + 1], pl[2 * e + 1]);
            }
#pragma unroll
            for (int j = 0; j < VT / 2; ++j) {
                uint32_t b[4];
                ldmatrix_x4_trans(b, v_base + (k * 16 * ldp + min(j, vpairs - 1) * 16) * 2);
                mma_bf16_16816(o[2 * j], ph, b[0], b[1]);
                mma_bf16_16816(o[2 * j + 1], ph, b[2], b[3]);
                mma_bf16_16816(o[2 * j], pl, b[0], b[1]);
                mma_bf16_16816(o[2 * j + 1], pl, b[2], b[3]);
            }
        }
    }
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 1);
        l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 2);
    }
    if constexpr (WP == 1) {
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            const int i = wr * 16 + h * 8 + (lane >> 2);
            if (i >= n_here) continue;
            const size_t pr = part_row(i);
            if ((lane & 3) == 0) { a.part.ml[2 * pr] = m_run[h] * 0.6931471805599453f; a.part.ml[2 * pr + 1] = l_run[h]; }
            float* po = a.part.o + pr * a.vdim;
#pragma unroll
            for (int j = 0; j < VT; ++j) {
                const int c = j * 8 + (lane & 3) * 2;
                if (c < a.vdim) po[c] = o[j][2 * h];
                if (c + 1 < a.vdim) po[c + 1] = o[j][2 * h + 1];
            }
        }
    } else {
        // the warps' positions meet in the ring's memory
        const int old = a.vd + 4;
        float* so = reinterpret_cast<float*>(skv);   // [warps][16][old]
#pragma unroll
        for (int h = 0; h < 2; ++h)
            if ((lane & 3) == 0) { s_ml[warp][h * 8 + (lane >> 2)][0] = m_run[h]; s_ml[warp][h * 8 + (lane >> 2)][1] = l_run[h]; }
        cp_async_wait<0>();
        __syncthreads();
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            const int i = h * 8 + (lane >> 2);
            float M = -INFINITY;
#pragma unroll
            for (int w = 0; w < kHmWarps; ++w) M = fmaxf(M, s_ml[w][i][0]);
            const float f = m_run[h] == -INFINITY ? 0.0f : exp2f(m_run[h] - M);
#pragma unroll
            for (int j = 0; j < VT; ++j)
                if (j * 8 < a.vd) *reinterpret_cast<float2*>(so + ((size_t)warp * 16 + i) * old + j * 8 + (lane & 3) * 2) = make_float2(o[j][2 * h] * f, o[j][2 * h + 1] * f);
        }
        __syncthreads();
        for (int i = tid; i < n_here * a.vdim; i += kHmThreads) {
            const int row = i / a.vdim, c = i % a.vdim;
            float v = 0.0f;
#pragma unroll
            for (int w = 0; w < kHmWarps; ++w) v += so[((size_t)w * 16 + row) * old + c];
            a.part.o[part_row(row) * a.vdim + c] = v;
        }
        if (tid < n_here) {
            float M = -INFINITY, L = 0.0f;
#pragma unroll
            for (int w = 0; w < kHmWarps; ++w) M = fmaxf(M, s_ml[w][tid][0]);
#pragma unroll
            for (int w = 0; w < kHmWarps; ++w)
                if (s_ml[w][tid][0] > -INFINITY) L += s_ml[w][tid][1] * exp2f(s_ml[w][tid][0] - M);
            float* ml = a.part.ml + 2 * part_row(tid);
            ml[0] = M * 0.6931471805599453f;
            ml[1] = L;
        }
    }
}

}  // namespace oxg4
