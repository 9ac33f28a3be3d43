// Kernels of models whose layers are listed one by one (csrc/layered.inl): recurrent mixers with a matrix state per
// head (lightning attention, retention, RWKV-style time mixing), token shift, grouped output norms with a gate, and
// attention over a paged cache of rows: multi-head latent attention, and grouped-query attention with a sink. They sit around the projections of gemv.cuh (one row, or f32
// weights) and tc_gemm.cuh (BF16 weights, many rows); the sandwich norms and the residual stream are those of
// rows_norm_kernel / the PRO_NORM prologue.
//
// Everything here computes in f32. Activations are rounded to BF16 only where they become the operand of a
// BF16 projection. "Split input": the consumer of a tcgen05 projection adds its K-split partials itself, in split
// order, so every reader takes (pointer, number of splits, distance between splits).
#pragma once
#include "batch_ops.cuh"
#include "common.cuh"
#include "gemv.cuh"

namespace oxg4 {

struct SplitIn {             // [splits][rows][ld] f32, columns start at `col`
    const float* p;
    int splits;
    size_t stride;           // elements between two splits
    int ld;
    DEVINL float at(int row, int col) const {
        const float* q = p + (size_t)row * ld + col;
        float t = q[0];
        for (int s = 1; s < splits; ++s) t += q[(size_t)s * stride];
        return t;
    }
};

// The rows of a pass as runs of consecutive tokens of one sequence (a decode step: one run of one token per
// sequence) and their positions.
struct RunRows {
    const int32_t* row0;     // [runs] first row
    const int32_t* n;        // [runs] rows
    const int32_t* pos;      // [R]
    const int32_t* seq;      // [R] or null: row r is sequence r
    const uint32_t* tok;     // [R]; kInactiveToken rows are left out
    DEVINL int seq_of(int row) const { return seq ? seq[row] : row; }
};

// The rows of a run, per_token of them per token, laid end to end and cut into tiles of `tile_rows`: run and first row
// (inside the run) of tile t over all runs, run -1 past the end. One warp.
DEVINL void find_row_tile(const RunRows& rows, int runs, int per_token, int tile_rows, int t, int& run, int& first) {
    const int lane = threadIdx.x & 31;
    int base = 0;
    run = -1;
    first = 0;
    for (int r0 = 0; r0 < runs && run < 0; r0 += 32) {
        const int r = r0 + lane;
        const int nt = r < runs ? (rows.n[r] * per_token + tile_rows - 1) / tile_rows : 0;
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
            first = (t - __shfl_sync(0xffffffffu, lo, src)) * tile_rows;
        }
        base += __shfl_sync(0xffffffffu, inc, 31);
    }
}

template <typename XT> DEVINL void store_act(XT* p, float v);
template <> DEVINL void store_act<float>(float* p, float v) { *p = v; }
template <> DEVINL void store_act<uint16_t>(uint16_t* p, float v) { *p = (uint16_t)f32_to_bf16_bits(v); }

// ---- token shift --------------------------------------------------------------------------------------------
// mix[s][r] = h_r + (h_(r-1) - h_r) * mu_s for S mixes; h_(r-1) is the previous row of the run, the sequence's shift
// state for the first row of a run, zero at position 0. grid (R), rows of H values (a multiple of 4).
template <typename XT>
__global__ void __launch_bounds__(256)
shift_mix_kernel(int R, int H, int S, const float* h, const float* state, const float* mu, RunRows rows, XT* mix) {
    pdl_wait();
    pdl_launch();
    const int r = blockIdx.x, s_ = rows.seq_of(r);
    const bool first = rows.seq == nullptr || r == 0 || rows.seq[r - 1] != s_;
    const float* prev = first ? state + (size_t)s_ * H : h + (size_t)(r - 1) * H;
    const bool zero = first && rows.pos[r] == 0;
    for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
        const float4 c = *reinterpret_cast<const float4*>(h + (size_t)r * H + i);
        float4 p = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (!zero) p = *reinterpret_cast<const float4*>(prev + i);
        for (int s = 0; s < S; ++s) {
            const float4 m = *reinterpret_cast<const float4*>(mu + (size_t)s * H + i);
            const float a = c.x + (p.x - c.x) * m.x, b = c.y + (p.y - c.y) * m.y, d = c.z + (p.z - c.z) * m.z,
                        e = c.w + (p.w - c.w) * m.w;
            XT* o = mix + ((size_t)s * R + r) * H + i;
            if constexpr (sizeof(XT) == 2) {
                *reinterpret_cast<uint2*>(o) = make_uint2(f32_to_bf16_bits(a) | (f32_to_bf16_bits(b) << 16),
                                                          f32_to_bf16_bits(d) | (f32_to_bf16_bits(e) << 16));
            } else {
                *reinterpret_cast<float4*>(o) = make_float4(a, b, d, e);
            }
        }
    }
}

// ---- per-channel decay of the time mixing -------------------------------------------------------------------
constexpr int kDecayRows = 8;
// out[r, n] = exp(-exp(W2[n, :] . tanh(low[r, :]) + w0[n])) for R rows and N channels; grid (ceil(N / 256), ceil(R / 8)), dynamic shared memory 8 * rank floats
template <typename WT>
__global__ void __launch_bounds__(256)
wkv_decay_kernel(int R, int N, int rank, SplitIn low, int col, const WT* w2, const float* w0, float* out) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    float* th = reinterpret_cast<float*>(smem_raw);
    pdl_wait();
    pdl_launch();
    const int r0 = blockIdx.y * kDecayRows, nr = min(kDecayRows, R - r0);
    for (int i = threadIdx.x; i < kDecayRows * rank; i += blockDim.x)
        th[i] = i / rank < nr ? tanhf(low.at(r0 + i / rank, col + i % rank)) : 0.0f;
    __syncthreads();
    const int n = blockIdx.x * 256 + threadIdx.x;
    if (n >= N) return;
    float t[kDecayRows];
#pragma unroll
    for (int q = 0; q < kDecayRows; ++q) t[q] = w0[n];
    constexpr int EPL = WTraits<WT>::EPL;
    if (rank % EPL == 0) {               // rows of W2 are whole 16-byte pieces
#pragma unroll 2
        for (int j = 0; j < rank; j += EPL) {
            const uint4 p = *reinterpret_cast<const uint4*>(w2 + (size_t)n * rank + j);
#pragma unroll
            for (int e = 0; e < EPL; ++e) {
                const float w = WTraits<WT>::elem(&p, e);
#pragma unroll
                for (int q = 0; q < kDecayRows; ++q) t[q] = fmaf(w, th[q * rank + j + e], t[q]);
            }
        }
    } else {
        for (int j = 0; j < rank; ++j) {
            const float w = WTraits<WT>::elem(w2, (size_t)n * rank + j);
#pragma unroll
            for (int q = 0; q < kDecayRows; ++q) t[q] = fmaf(w, th[q * rank + j], t[q]);
        }
    }
#pragma unroll
    for (int q = 0; q < kDecayRows; ++q)
        if (q < nr) out[(size_t)(r0 + q) * N + n] = expf(-expf(t[q]));
}

// ---- recurrence ---------------------------------------------------------------------------------------------
// Per head a state S [dim, vdim] in f32, walked token by token:
//   REC_LIGHTNING  q, k, v = silu(.);  S = decay_h S + k v^T;  o = S^T q
//   REC_RETENTION  the same recurrence; q and k are rotated (channel i with i + rot_dims / 2) and k is scaled instead
//   REC_WKV        o = (S + diag(u) k v^T)^T r;  S = diag(w) S + k v^T, w per token and key channel
// The bonus term is v * sum_k r_k u_k k_k, one scalar per token and head.
// recur_kernel: decode steps, and time mixing in prompts. Grid (heads, slices of vdim, runs). A thread owns KPT key channels of two value columns; the KS threads that share
// a column are neighbouring lanes. Tokens are staged in shared memory in tiles, activations applied on
// the way; the dot products of up to 8 tokens are reduced across the KS lanes together.
// State in memory: [sequence][head][vdim][dim]. At position 0 the state starts at zero whatever the memory holds.
//
// Prompts with fixed decays (LIGHTNING, RETENTION) go through fixed_recur_kernel: a run is cut into blocks of kRecBlock tokens
// that are walked side by side, every block but the first from a zero state, and recur_join_kernel adds what the state at a
// block's start contributes: o_t += decay^(t + 1) S_start^T q_t for the block's t-th token, S_start = sum of the earlier
// blocks' end states times the decay in between. End states lie in slots of their own, 2 * (first row / kRecBlock), plus one
// for a block that is not full: full blocks begin kRecBlock rows apart, and a last, shorter block follows a full one.
enum { REC_LIGHTNING = 0, REC_WKV = 1, REC_RETENTION = 2 };
constexpr int kRecThreads = 128;
constexpr int kRecCols = 2;              // value columns per thread
constexpr int kRecBlock = 64;            // tokens of a block
constexpr int kRecMaxBlocks = 4;         // blocks of the longest run (a pass carries at most 256 rows)
__host__ __device__ constexpr int rec_tile(int dp) { return dp <= 128 ? 16 : dp <= 256 ? 8 : 4; }   // tokens staged at a time

struct RecurArgs {
    SplitIn in;                          // fused input projection
    int c_q, c_k, c_v;                   // first columns of q (r), k and v, head by head
    int heads, dim, vdim;
    const float* decay;                  // LIGHTNING, RETENTION: [heads]
    const float2* freq;                  // RETENTION: [rot_dims / 2] turns per position, high and low part
    int rot_dims;
    float k_scale;
    const float* u;                      // WKV: [heads, dim]
    const float* w;                      // WKV: [R, heads * dim] decays, or null: computed here (runs of one token)
    int c_low, rank;                     //   from the low-rank columns
    const void* w2;                      //   [heads * dim, rank]
    const float* w0;                     //   [heads * dim]
    float* state;
    float* block_state;                  // fixed_recur_kernel: [slots][heads][vdim][dim]
    float* block_q;                      //   [R, heads * dim] activated queries for recur_join_kernel
    int runs;
    RunRows rows;
    float* out;                          // [R, ld_out]
    int ld_out;
    // token-shift state: the normed input of the run's last row, copied by one CTA per run
    const float* shift_src;              // [R, shift_n] or null
    float* shift_dst;                    // [sequences, shift_n]
    int shift_n;
};

// Sums acc[0 .. N) over the KS neighbouring lanes of a column, halving the tokens a lane keeps at every step: lane ks ends
// with the totals of tokens `first` .. `first + left - 1` in acc[0 .. left), left = max(1, N / KS).
template <int N, int KS>
DEVINL void column_reduce(float (&acc)[N], int ks, int& first) {
    int left = N;
    first = 0;
#pragma unroll
    for (int o = KS / 2; o > 0; o >>= 1) {
        if (left > 1) {
            left /= 2;
            const bool up = (ks & o) != 0;
#pragma unroll
            for (int t = 0; t < N / 2; ++t)
                if (t < left) {
                    const float keep = up ? acc[t + left] : acc[t], send = up ? acc[t] : acc[t + left];
                    acc[t] = keep + __shfl_xor_sync(0xffffffffu, send, o);
                }
            if (up) first += left;
        } else {
            acc[0] += __shfl_xor_sync(0xffffffffu, acc[0], o);
        }
    }
}

// TILE: tokens staged at a time; 1 for decode steps (row r is sequence r's one token). Tiles of longer runs are
// double-buffered: the next tile's values are fetched into registers while the current one is walked. A thread's key
// channels come in groups of four, KS * 4 apart, so that the lanes of a column read neighbouring 16-byte pieces.
// sine and cosine of the angle at `pos`: p * (hi + lo) turns to more than f32, whole turns taken off exactly
DEVINL void rotation(int pos, float2 freq, float& sn, float& cs) {
    const float p = (float)pos, a = p * freq.x, e = fmaf(p, freq.x, -a) + p * freq.y;
    sincospif(2.0f * ((a - rintf(a)) + e), &sn, &cs);
}

struct RecBlock {
    int row0, n, first;                  // rows, place of the first one in its run
    bool split, last;                    // the run has more than one block; this is its last one
    size_t slot;
};
DEVINL bool find_block(const RecurArgs& a, int t, RecBlock& b) {
    __shared__ int s_run, s_first;
    if (threadIdx.x < 32) {
        int run, first;
        find_row_tile(a.rows, a.runs, 1, kRecBlock, t, run, first);
        if (threadIdx.x == 0) { s_run = run; s_first = first; }
    }
    __syncthreads();
    if (s_run < 0) return false;
    b.first = s_first;
    b.row0 = a.rows.row0[s_run] + b.first;
    b.n = min(kRecBlock, a.rows.n[s_run] - b.first);
    b.split = a.rows.n[s_run] > kRecBlock;
    b.last = b.first + b.n == a.rows.n[s_run];
    b.slot = 2 * (size_t)(b.row0 / kRecBlock) + (b.n < kRecBlock ? 1 : 0);
    return true;
}

template <int KIND, typename WT, int KS, int KPT, int TILE>
__global__ void __launch_bounds__(kRecThreads) recur_kernel(const RecurArgs a) {
    constexpr bool WKV = KIND == REC_WKV, RET = KIND == REC_RETENTION;
    constexpr int DP = KS * KPT;         // key channels, padded
    constexpr int VG = kRecThreads / KS; // threads along the value columns
    constexpr int VS = VG * kRecCols;    // value columns of this CTA
    constexpr int NK = (TILE * DP + kRecThreads - 1) / kRecThreads, NV = (TILE * VS + kRecThreads - 1) / kRecThreads;
    constexpr int TB = TILE < 8 ? TILE : 8;
    constexpr int TPAD = (TILE + 3) / 4 * 4;
    constexpr int BUF = TILE * DP * (WKV ? 3 : 2) + TILE * VS + TPAD;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    float* bufs = reinterpret_cast<float*>(smem_raw);        // [2 (1 for TILE 1)][q | k | w (WKV) | v | bonus (WKV)]
    float* su = bufs + (TILE == 1 ? 1 : 2) * BUF;            // WKV: [DP] u of this head, then [rank] for one-token runs
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int hd = blockIdx.x, v0 = blockIdx.y * VS, run = blockIdx.z;
    const int ks = tid % KS, vg = tid / KS;
    const int hk = hd * a.dim, hv = hd * a.vdim;
    auto channel = [&](int i) { return (i / 4) * (KS * 4) + ks * 4 + i % 4; };
    if constexpr (WKV)
        for (int k = tid; k < DP; k += kRecThreads) su[k] = k < a.dim ? a.u[hk + k] : 0.0f;
    pdl_wait();
    pdl_launch();
    const int row0 = TILE == 1 ? run : a.rows.row0[run], n = TILE == 1 ? 1 : a.rows.n[run];
    const int seq = a.rows.seq_of(row0);
    const uint32_t tok = a.rows.tok[row0];
    const int pos = a.rows.pos[row0];
    float* st = a.state + (((size_t)seq * a.heads + hd) * a.vdim + v0 + vg) * a.dim;     // column j: VG * dim further
    float S[kRecCols][KPT];
#pragma unroll
    for (int j = 0; j < kRecCols; ++j) {
        const bool have = v0 + vg + j * VG < a.vdim;
        const float* sj = st + (size_t)j * VG * a.dim;
        if (a.dim % 4 == 0) {
#pragma unroll
            for (int i = 0; i < KPT; i += 4) {
                float4 x = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                if (have && channel(i) < a.dim) x = *reinterpret_cast<const float4*>(sj + channel(i));
                S[j][i] = x.x; S[j][i + 1] = x.y; S[j][i + 2] = x.z; S[j][i + 3] = x.w;
            }
        } else {
#pragma unroll
            for (int i = 0; i < KPT; ++i) S[j][i] = (have && channel(i) < a.dim) ? sj[channel(i)] : 0.0f;
        }
    }
    float fq[NK], fk[NK], fw[WKV ? NK : 1], fv[NV];
    auto fetch = [&](int t0) {           // values of the tile at t0, zero past the run and past the key channels
        const float* base = a.in.p + (size_t)(row0 + t0) * a.in.ld;
#pragma unroll
        for (int j = 0; j < NK; ++j) {
            const int i = tid + j * kRecThreads, t = i / DP, k = i % DP;
            const bool ok = i < TILE * DP && t0 + t < n && k < a.dim;
            const float* p = base + (size_t)t * a.in.ld + hk + k;
            fq[j] = ok ? p[a.c_q] : 0.0f;
            fk[j] = ok ? p[a.c_k] : 0.0f;
            if constexpr (WKV) fw[j] = ok && a.w != nullptr ? a.w[(size_t)(row0 + t0 + t) * a.heads * a.dim + hk + k] : 0.0f;
        }
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int i = tid + j * kRecThreads, t = i / VS, c = v0 + i % VS;
            fv[j] = (i < TILE * VS && t0 + t < n && c < a.vdim) ? base[(size_t)t * a.in.ld + a.c_v + hv + c] : 0.0f;
        }
        for (int s = 1; s < a.in.splits; ++s) {
            const float* part = base + s * a.in.stride;
#pragma unroll
            for (int j = 0; j < NK; ++j) {
                const int i = tid + j * kRecThreads, t = i / DP, k = i % DP;
                if (i < TILE * DP && t0 + t < n && k < a.dim) {
                    fq[j] += part[(size_t)t * a.in.ld + a.c_q + hk + k];
                    fk[j] += part[(size_t)t * a.in.ld + a.c_k + hk + k];
                }
            }
#pragma unroll
            for (int j = 0; j < NV; ++j) {
                const int i = tid + j * kRecThreads, t = i / VS, c = v0 + i % VS;
                if (i < TILE * VS && t0 + t < n && c < a.vdim) fv[j] += part[(size_t)t * a.in.ld + a.c_v + hv + c];
            }
        }
    };
    fetch(0);
    if (tok == kInactiveToken) return;
    if (pos == 0) {
#pragma unroll
        for (int j = 0; j < kRecCols; ++j)
#pragma unroll
            for (int i = 0; i < KPT; ++i) S[j][i] = 0.0f;
    }
    if (a.shift_src != nullptr && hd == 0 && blockIdx.y == 0)
        for (int i = tid; i < a.shift_n; i += kRecThreads)
            a.shift_dst[(size_t)seq * a.shift_n + i] = a.shift_src[(size_t)(row0 + n - 1) * a.shift_n + i];
    const float dh = WKV ? 0.0f : a.decay[hd];
    int parity = 0;
    for (int t0 = 0; t0 < n; t0 += TILE) {
        const int nt = min(TILE, n - t0);
        float* sq = bufs + parity * BUF;
        float *sk = sq + TILE * DP, *sw = sk + TILE * DP, *sv = sw + (WKV ? TILE * DP : 0), *sb = sv + TILE * VS;
#pragma unroll
        for (int j = 0; j < NK; ++j) {
            const int i = tid + j * kRecThreads;
            if (i < TILE * DP) {
                sq[i] = WKV || RET ? fq[j] : silu(fq[j]);
                sk[i] = WKV ? fk[j] : RET ? fk[j] * a.k_scale : silu(fk[j]);
                if constexpr (WKV) sw[i] = fw[j];
            }
        }
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int i = tid + j * kRecThreads;
            if (i < TILE * VS) sv[i] = WKV || RET ? fv[j] : silu(fv[j]);
        }
        if (t0 + TILE < n) fetch(t0 + TILE);
        if constexpr (RET) {
            __syncthreads();
            const int half = a.rot_dims / 2;
            for (int i = tid; i < nt * half; i += kRecThreads) {
                const int t = i / half, d = i % half;
                float sn, cs;
                rotation(pos + t0 + t, a.freq[d], sn, cs);
                float *q = sq + t * DP + d, *k = sk + t * DP + d;
                const float qu = q[0], qv = q[half], ku = k[0], kv = k[half];
                q[0] = qu * cs - qv * sn;
                q[half] = qv * cs + qu * sn;
                k[0] = ku * cs - kv * sn;
                k[half] = kv * cs + ku * sn;
            }
        }
        if constexpr (WKV && TILE == 1) {
            if (a.w == nullptr) {                            // decay of this head's channels, four lanes per channel
                float* th = su + DP;                         // [rank]
                for (int j = tid; j < a.rank; j += kRecThreads) th[j] = tanhf(a.in.at(row0, a.c_low + j));
                __syncthreads();
                for (int k0 = 0; k0 < a.dim; k0 += kRecThreads / 4) {
                    const int k = k0 + (tid >> 2);
                    float t = 0.0f;
                    if (k < a.dim)
#pragma unroll 8
                        for (int j = tid & 3; j < a.rank; j += 4) t = fmaf(WTraits<WT>::elem(a.w2, (size_t)(hk + k) * a.rank + j), th[j], t);
                    t += __shfl_xor_sync(0xffffffffu, t, 1);
                    t += __shfl_xor_sync(0xffffffffu, t, 2);
                    if (k < a.dim && (tid & 3) == 0) sw[k] = expf(-expf(t + a.w0[hk + k]));
                }
            }
        }
        __syncthreads();
        if constexpr (WKV && TILE > 1) {                     // bonus of every token: sum over k of r u k
            for (int t = warp; t < nt; t += kRecThreads / 32) {
                float b = 0.0f;
                for (int k = lane; k < DP; k += 32) b += sq[t * DP + k] * su[k] * sk[t * DP + k];
                b = warp_sum(b);
                if (lane == 0) sb[t] = b;
            }
            __syncthreads();
        }
        for (int tb = 0; tb < nt; tb += TB) {
            float acc[kRecCols][TB];
#pragma unroll
            for (int t = 0; t < TB; ++t) {
#pragma unroll
                for (int j = 0; j < kRecCols; ++j) acc[j][t] = 0.0f;
                if (tb + t >= nt) continue;
                const float* q = sq + (tb + t) * DP + ks * 4;
                const float* k = sk + (tb + t) * DP + ks * 4;
                const float* w = sw + (tb + t) * DP + ks * 4;
                float x[kRecCols];
#pragma unroll
                for (int j = 0; j < kRecCols; ++j) x[j] = sv[(tb + t) * VS + vg + j * VG];
#pragma unroll
                for (int i = 0; i < KPT; i += 4) {
                    const float4 q4 = *reinterpret_cast<const float4*>(q + i * KS), k4 = *reinterpret_cast<const float4*>(k + i * KS);
                    const float qe[4] = {q4.x, q4.y, q4.z, q4.w}, ke[4] = {k4.x, k4.y, k4.z, k4.w};
                    if constexpr (!WKV) {
#pragma unroll
                        for (int j = 0; j < kRecCols; ++j)
#pragma unroll
                            for (int e = 0; e < 4; ++e) {
                                S[j][i + e] = fmaf(dh, S[j][i + e], ke[e] * x[j]);
                                acc[j][t] = fmaf(qe[e], S[j][i + e], acc[j][t]);
                            }
                    } else {
                        const float4 w4 = *reinterpret_cast<const float4*>(w + i * KS);
                        const float we[4] = {w4.x, w4.y, w4.z, w4.w};
                        if constexpr (TILE == 1) {
                            const float4 u4 = *reinterpret_cast<const float4*>(su + ks * 4 + i * KS);
                            const float ue[4] = {u4.x, u4.y, u4.z, u4.w};
#pragma unroll
                            for (int j = 0; j < kRecCols; ++j)
#pragma unroll
                                for (int e = 0; e < 4; ++e) acc[j][t] = fmaf(qe[e] * ue[e] * ke[e], x[j], acc[j][t]);
                        }
#pragma unroll
                        for (int j = 0; j < kRecCols; ++j)
#pragma unroll
                            for (int e = 0; e < 4; ++e) {
                                acc[j][t] = fmaf(qe[e], S[j][i + e], acc[j][t]);
                                S[j][i + e] = fmaf(we[e], S[j][i + e], ke[e] * x[j]);
                            }
                    }
                }
            }
            constexpr int LEFT = TB / KS > 0 ? TB / KS : 1;
            // with more lanes than tokens the lanes that differ in the low bits hold the same total: one of them stores
            const bool owner = KS <= TB || ks % (KS / TB > 0 ? KS / TB : 1) == 0;
#pragma unroll
            for (int j = 0; j < kRecCols; ++j) {
                int first;
                column_reduce<TB, KS>(acc[j], ks, first);
                const int c = vg + j * VG;
                if (v0 + c < a.vdim && owner) {
#pragma unroll
                    for (int t = 0; t < LEFT; ++t) {
                        const int tt = tb + first + t;
                        if (tt < nt) {
                            float o = acc[j][t];
                            if constexpr (WKV && TILE > 1) o = fmaf(sb[tt], sv[tt * VS + c], o);
                            a.out[(size_t)(row0 + t0 + tt) * a.ld_out + hv + v0 + c] = o;
                        }
                    }
                }
            }
        }
        parity ^= 1;
    }
#pragma unroll
    for (int j = 0; j < kRecCols; ++j) {
        if (v0 + vg + j * VG >= a.vdim) continue;
        float* sj = st + (size_t)j * VG * a.dim;
        if (a.dim % 4 == 0) {
#pragma unroll
            for (int i = 0; i < KPT; i += 4)
                if (channel(i) < a.dim) *reinterpret_cast<float4*>(sj + channel(i)) = make_float4(S[j][i], S[j][i + 1], S[j][i + 2], S[j][i + 3]);
        } else {
#pragma unroll
            for (int i = 0; i < KPT; ++i)
                if (channel(i) < a.dim) sj[channel(i)] = S[j][i];
        }
    }
}

// two f32 multiply-adds or products per instruction
DEVINL uint64_t fma_f32x2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
DEVINL uint64_t mul_f32x2(uint64_t a, uint64_t b) {
    uint64_t d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
DEVINL uint64_t pack_f32x2(float x, float y) {
    uint64_t d;
    asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(x), "f"(y));
    return d;
}
DEVINL float2 unpack_f32x2(uint64_t v) {
    float2 d;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(d.x), "=f"(d.y) : "l"(v));
    return d;
}

// tokens staged at a time: 37 KB of q, k and v at most, so that six CTAs fit on an SM
__host__ __device__ constexpr int rec_stage(int dp) { return dp <= 128 ? 32 : dp <= 256 ? 16 : 8; }
__host__ __device__ constexpr size_t fixed_recur_smem(int ks, int kpt) { return sizeof(float) * rec_stage(ks * kpt) * (2 * ks * kpt + kRecThreads / ks * kRecCols); }

// One block of a run per CTA: grid (heads, slices of vdim, blocks), threads and key channels as in recur_kernel, two channels
// per register pair. The loops are kept short on purpose: a launch of a few thousand instructions per warp spends its time on
// fetching code that it runs once.
template <int KIND, int KS, int KPT>
__global__ void __launch_bounds__(kRecThreads, KPT <= 16 && KS <= 8 ? 5 : 3) fixed_recur_kernel(const RecurArgs a) {
    constexpr int DP = KS * KPT, VG = kRecThreads / KS, VS = VG * kRecCols, ROWS = rec_stage(DP);
    constexpr int NV = 2 * kRecCols;     // dot products of two tokens
    static_assert(kRecCols == 2, "two value columns per thread");
    constexpr int LD = 2 * DP + VS, L4 = LD / 4;             // a staged token: q | k | v
    extern __shared__ __align__(16) unsigned char smem_raw[];
    float* st = reinterpret_cast<float*>(smem_raw);          // [ROWS][LD]
    const int tid = threadIdx.x, hd = blockIdx.x, v0 = blockIdx.y * VS, ks = tid % KS, vg = tid / KS;
    const int hk = hd * a.dim, hv = hd * a.vdim;
    auto channel = [&](int i) { return (i / 4) * (KS * 4) + ks * 4 + i % 4; };
    RecBlock b;                                              // rows and positions were there before the preceding kernel
    const bool any = find_block(a, blockIdx.z, b);
    const int seq = any ? a.rows.seq_of(b.row0) : 0, pos = any ? a.rows.pos[b.row0] : 0;
    pdl_wait();
    pdl_launch();
    if (!any) return;
    const size_t mine = ((size_t)hd * a.vdim + v0 + vg) * a.dim, all = (size_t)a.heads * a.vdim * a.dim;
    uint64_t S[kRecCols][KPT / 2];
    const bool resume = b.first == 0 && pos > 0, vec = a.dim % 4 == 0;
#pragma unroll
    for (int j = 0; j < kRecCols; ++j) {
        const bool have = resume && v0 + vg + j * VG < a.vdim;
        const float* sj = a.state + seq * all + mine + (size_t)j * VG * a.dim;
#pragma unroll
        for (int i = 0; i < KPT; i += 4) {
            const int c = channel(i);
            float4 x = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (have && c < a.dim) {
                if (vec) x = *reinterpret_cast<const float4*>(sj + c);
                else x = make_float4(sj[c], c + 1 < a.dim ? sj[c + 1] : 0.0f, c + 2 < a.dim ? sj[c + 2] : 0.0f, c + 3 < a.dim ? sj[c + 3] : 0.0f);
            }
            S[j][i / 2] = pack_f32x2(x.x, x.y);
            S[j][i / 2 + 1] = pack_f32x2(x.z, x.w);
        }
    }
    const float dh = a.decay[hd], kf = a.k_scale;
    const bool vec_in = vec && (a.vdim & 3) == 0 && ((a.c_q | a.c_k | a.c_v | a.in.ld) & 3) == 0;
    auto place = [&](int c, bool& ok) {                      // column of the input projection for column c of a staged token
        const int d = c < DP ? c : c < 2 * DP ? c - DP : c - 2 * DP;
        ok = c < 2 * DP ? d < a.dim : v0 + d < a.vdim;
        return c < DP ? a.c_q + hk + d : c < 2 * DP ? a.c_k + hk + d : a.c_v + hv + v0 + d;
    };
    auto act = [&](float x, int c) { return KIND == REC_LIGHTNING ? silu(x) : c >= DP && c < 2 * DP ? x * kf : x; };
#pragma unroll 1
    for (int t0 = 0; t0 < b.n; t0 += ROWS) {
        const int n = min(ROWS, b.n - t0), row = b.row0 + t0;
        if (t0 > 0) __syncthreads();
        if (vec_in) {
            constexpr int U = 6;                             // loads in flight per thread
#pragma unroll 1
            for (int i0 = tid; i0 < ROWS * L4; i0 += U * kRecThreads) {
                float4 v[U];
#pragma unroll
                for (int u = 0; u < U; ++u) v[u] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                const float* p = a.in.p + (size_t)row * a.in.ld;
#pragma unroll 1
                for (int s = 0; s < a.in.splits; ++s, p += a.in.stride) {
                    float4 w[U];
#pragma unroll
                    for (int u = 0; u < U; ++u) {
                        const int i = i0 + u * kRecThreads, t = i / L4;
                        bool ok;
                        const int c = place(i % L4 * 4, ok);
                        w[u] = ok && t < n ? __ldcg(reinterpret_cast<const float4*>(p + (size_t)t * a.in.ld + c)) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                    }
#pragma unroll
                    for (int u = 0; u < U; ++u) { v[u].x += w[u].x; v[u].y += w[u].y; v[u].z += w[u].z; v[u].w += w[u].w; }
                }
#pragma unroll
                for (int u = 0; u < U; ++u) {
                    const int i = i0 + u * kRecThreads, c = i % L4 * 4;
                    if (i < ROWS * L4) *reinterpret_cast<float4*>(st + 4 * i) = make_float4(act(v[u].x, c), act(v[u].y, c), act(v[u].z, c), act(v[u].w, c));
                }
            }
        } else {
#pragma unroll 1
            for (int i = tid; i < ROWS * LD; i += kRecThreads) {
                bool ok;
                const int t = i / LD, c = i % LD, from = place(c, ok);
                st[i] = ok && t < n ? act(a.in.at(row + t, from), c) : 0.0f;
            }
        }
        if constexpr (KIND == REC_RETENTION) {
            __syncthreads();
            const int half = a.rot_dims / 2;
#pragma unroll 1
            for (int i = tid; i < n * half; i += kRecThreads) {
                const int t = i / half, d = i % half;
                float sn, cs;
                rotation(pos + t0 + t, a.freq[d], sn, cs);
                float *q = st + t * LD + d, *k = q + DP;
                const float qu = q[0], qv = q[half], ku = k[0], kv = k[half];
                q[0] = qu * cs - qv * sn;
                q[half] = qv * cs + qu * sn;
                k[0] = ku * cs - kv * sn;
                k[half] = kv * cs + ku * sn;
            }
        }
        __syncthreads();
        if (blockIdx.y == 0 && b.first > 0) {
            float* to = a.block_q + (size_t)row * a.heads * a.dim + hk;
            if (vec) {
#pragma unroll 4
                for (int i = tid; i < n * (DP / 4); i += kRecThreads) {
                    const int t = i / (DP / 4), d = i % (DP / 4) * 4;
                    if (d < a.dim) *reinterpret_cast<float4*>(to + (size_t)t * a.heads * a.dim + d) = *reinterpret_cast<const float4*>(st + t * LD + d);
                }
            } else {
#pragma unroll 1
                for (int i = tid; i < n * DP; i += kRecThreads)
                    if (i % DP < a.dim) to[(size_t)(i / DP) * a.heads * a.dim + i % DP] = st[i / DP * LD + i % DP];
            }
        }
#pragma unroll 1
        for (int t = 0; t < n; t += 2) {
            uint64_t acc[2][kRecCols] = {};
#pragma unroll
            for (int u = 0; u < 2; ++u) {                    // a second token that is not there (zeros) keeps the state
                const float *q = st + (t + u) * LD + ks * 4, *k = q + DP, *v = st + (t + u) * LD + 2 * DP + vg;
                const float f = t + u < n ? dh : 1.0f;
                const uint64_t d2 = pack_f32x2(f, f);
                uint64_t x[kRecCols];
#pragma unroll
                for (int j = 0; j < kRecCols; ++j) x[j] = pack_f32x2(v[j * VG], v[j * VG]);
#pragma unroll
                for (int i = 0; i < KPT; i += 4) {
                    const ulonglong2 q4 = *reinterpret_cast<const ulonglong2*>(q + i * KS), k4 = *reinterpret_cast<const ulonglong2*>(k + i * KS);
#pragma unroll
                    for (int j = 0; j < kRecCols; ++j) {
                        uint64_t &s0 = S[j][i / 2], &s1 = S[j][i / 2 + 1];
                        s0 = fma_f32x2(d2, s0, mul_f32x2(k4.x, x[j]));
                        s1 = fma_f32x2(d2, s1, mul_f32x2(k4.y, x[j]));
                        acc[u][j] = fma_f32x2(q4.x, s0, acc[u][j]);
                        acc[u][j] = fma_f32x2(q4.y, s1, acc[u][j]);
                    }
                }
            }
            float o[NV];
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const float2 v = unpack_f32x2(acc[i / kRecCols][i % kRecCols]);
                o[i] = v.x + v.y;
            }
            int first;
            column_reduce<NV, KS>(o, ks, first);             // this lane's total is number `first`
            const int u = first / kRecCols, c = vg + first % kRecCols * VG;
            if (t + u < n && v0 + c < a.vdim && (KS <= NV || ks % (KS > NV ? KS / NV : 1) == 0))
                a.out[(size_t)(row + t + u) * a.ld_out + hv + v0 + c] = o[0];
        }
    }
    float* end = (b.split ? a.block_state + b.slot * all : a.state + seq * all) + mine;
#pragma unroll
    for (int j = 0; j < kRecCols; ++j) {
        if (v0 + vg + j * VG >= a.vdim) continue;
        float* sj = end + (size_t)j * VG * a.dim;
#pragma unroll
        for (int i = 0; i < KPT; i += 4) {
            const int c = channel(i);
            const float2 x = unpack_f32x2(S[j][i / 2]), y = unpack_f32x2(S[j][i / 2 + 1]);
            if (c >= a.dim) continue;
            if (vec) {
                *reinterpret_cast<float4*>(sj + c) = make_float4(x.x, x.y, y.x, y.y);
            } else {
                sj[c] = x.x;
                if (c + 1 < a.dim) sj[c + 1] = x.y;
                if (c + 2 < a.dim) sj[c + 2] = y.x;
                if (c + 3 < a.dim) sj[c + 3] = y.y;
            }
        }
    }
}

// Adds the start states' share to the outputs of the blocks behind the first one of a run and stores the run's end state.
// Grid (heads, slices of kJoinCols value columns, blocks); a thread owns 4 tokens x 4 value columns. dynamic shared memory:
// join_smem(dim).
constexpr int kJoinCols = 32, kJoinThreads = kRecBlock / 4 * (kJoinCols / 4);
__host__ __device__ constexpr int join_ld(int dim) { return (dim + 3) / 4 * 4 + 4; }     // neighbouring rows start 4 banks apart at dim 32, 64, ...
__host__ __device__ constexpr size_t join_smem(int dim) { return sizeof(float) * join_ld(dim) * (kRecBlock + kJoinCols); }
__global__ void __launch_bounds__(kJoinThreads) recur_join_kernel(const RecurArgs a) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int tid = threadIdx.x, hd = blockIdx.x, v0 = blockIdx.y * kJoinCols, nv = min(kJoinCols, a.vdim - v0);
    const int dim = a.dim, ld = join_ld(dim), d4 = (ld - 4) / 4;
    float* sq = reinterpret_cast<float*>(smem_raw);          // [kRecBlock][ld] queries
    float* ss = sq + (size_t)kRecBlock * ld;                 // [kJoinCols][ld] state at the block's start
    __shared__ float pw[kRecBlock + 1];                      // powers of the decay
    const float dh = a.decay[hd];
    if (tid <= kRecBlock) pw[tid] = powf(dh, (float)tid);
    RecBlock b;
    const bool mine_to_do = find_block(a, blockIdx.z, b) && b.first > 0;
    const int seq = mine_to_do ? a.rows.seq_of(b.row0) : 0;
    pdl_wait();
    pdl_launch();
    if (!mine_to_do) return;
    __syncthreads();
    // the earlier blocks of the run are full and lie one behind the other
    const size_t all = (size_t)a.heads * a.vdim * dim, here = ((size_t)hd * a.vdim + v0) * dim;
    const float* e0 = a.block_state + 2 * (size_t)((b.row0 - b.first) / kRecBlock) * all + here;
    const float* mine = a.block_state + b.slot * all + here;
    float* st = a.state + seq * all + here;
    const int earlier = b.first / kRecBlock;
    const float* q_in = a.block_q + (size_t)b.row0 * a.heads * dim + hd * dim;
    const float p = pw[kRecBlock], pn = pw[b.n];
    if (dim % 4 == 0) {
        const float4 none = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        constexpr int U = 8, W = 2;                          // loads in flight per thread: U, W * kRecMaxBlocks
#pragma unroll 1
        for (int i0 = tid; i0 < kRecBlock * d4; i0 += U * kJoinThreads) {
            float4 v[U];
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const int i = i0 + u * kJoinThreads, t = i / d4, d = i % d4 * 4;
                v[u] = t < b.n ? __ldcg(reinterpret_cast<const float4*>(q_in + (size_t)t * a.heads * dim + d)) : none;
            }
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const int i = i0 + u * kJoinThreads, t = i / d4;
                if (t < kRecBlock) *reinterpret_cast<float4*>(sq + t * ld + i % d4 * 4) = v[u];
            }
        }
#pragma unroll 1
        for (int i0 = tid; i0 < kJoinCols * d4; i0 += W * kJoinThreads) {
            float4 e[W][kRecMaxBlocks];                      // earlier blocks' end states, then this one's
#pragma unroll
            for (int u = 0; u < W; ++u) {
                const int i = i0 + u * kJoinThreads, c = i / d4;
                const size_t at = (size_t)4 * i;
#pragma unroll
                for (int j = 0; j < kRecMaxBlocks - 1; ++j)
                    e[u][j] = c < nv && j < earlier ? __ldcg(reinterpret_cast<const float4*>(e0 + 2 * j * all + at)) : none;
                e[u][kRecMaxBlocks - 1] = c < nv && b.last ? __ldcg(reinterpret_cast<const float4*>(mine + at)) : none;
            }
#pragma unroll
            for (int u = 0; u < W; ++u) {
                const int i = i0 + u * kJoinThreads, c = i / d4;
                if (c >= kJoinCols) continue;
                float4 s = none;
#pragma unroll
                for (int j = 0; j < kRecMaxBlocks - 1; ++j) {
                    const float f = j < earlier ? p : 1.0f;
                    s = make_float4(fmaf(s.x, f, e[u][j].x), fmaf(s.y, f, e[u][j].y), fmaf(s.z, f, e[u][j].z), fmaf(s.w, f, e[u][j].w));
                }
                *reinterpret_cast<float4*>(ss + c * ld + i % d4 * 4) = s;
                const float4 m = e[u][kRecMaxBlocks - 1];
                if (c < nv && b.last)
                    *reinterpret_cast<float4*>(st + (size_t)4 * i) = make_float4(fmaf(s.x, pn, m.x), fmaf(s.y, pn, m.y), fmaf(s.z, pn, m.z), fmaf(s.w, pn, m.w));
            }
        }
    } else {
#pragma unroll 1
        for (int i = tid; i < kRecBlock * ld; i += kJoinThreads) {
            const int t = i / ld, d = i % ld;
            sq[i] = t < b.n && d < dim ? __ldcg(q_in + (size_t)t * a.heads * dim + d) : 0.0f;
        }
#pragma unroll 1
        for (int i = tid; i < kJoinCols * ld; i += kJoinThreads) {
            const int c = i / ld, d = i % ld;
            const size_t at = (size_t)c * dim + d;
            float s = 0.0f;
            if (c < nv && d < dim) {
                for (int j = 0; j < earlier; ++j) s = fmaf(s, p, __ldcg(e0 + 2 * j * all + at));
                if (b.last) st[at] = fmaf(s, pn, __ldcg(mine + at));
            }
            ss[i] = s;
        }
    }
    __syncthreads();
    // tokens tg + 16 u, columns cg + 8 v: the rows that a warp reads together are neighbours
    constexpr int TG = kRecBlock / 4, CG = kJoinCols / 4;
    const int tg = tid / CG, cg = tid % CG;
    float acc[4][4] = {};
#pragma unroll 2
    for (int d = 0; d < 4 * d4; d += 4) {
        float4 q[4], x[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            q[u] = *reinterpret_cast<const float4*>(sq + (tg + TG * u) * ld + d);
            x[u] = *reinterpret_cast<const float4*>(ss + (cg + CG * u) * ld + d);
        }
#pragma unroll
        for (int u = 0; u < 4; ++u)
#pragma unroll
            for (int v = 0; v < 4; ++v)
                acc[u][v] = fmaf(q[u].w, x[v].w, fmaf(q[u].z, x[v].z, fmaf(q[u].y, x[v].y, fmaf(q[u].x, x[v].x, acc[u][v]))));
    }
    float* out = a.out + (size_t)b.row0 * a.ld_out + hd * a.vdim + v0;
    float o[4][4];
#pragma unroll
    for (int u = 0; u < 4; ++u)
#pragma unroll
        for (int v = 0; v < 4; ++v)
            o[u][v] = tg + TG * u < b.n && cg + CG * v < nv ? out[(size_t)(tg + TG * u) * a.ld_out + cg + CG * v] : 0.0f;
#pragma unroll
    for (int u = 0; u < 4; ++u)
#pragma unroll
        for (int v = 0; v < 4; ++v)
            if (tg + TG * u < b.n && cg + CG * v < nv) out[(size_t)(tg + TG * u) * a.ld_out + cg + CG * v] = fmaf(pw[tg + TG * u + 1], acc[u][v], o[u][v]);
}

// ---- output norm and gate of a mixer ------------------------------------------------------------------------
// Further columns of an output projection's input, from `at` on: the feed-forward's activations where mixer and
// feed-forward share the projection. In f32 multi-row passes they are finished values; behind a tcgen05 projection
// alternately gate and up values, `act` and product still to come. Slices of kTailCols columns.
constexpr int kTailCols = 1024;
struct OutTail {
    SplitIn in;
    int col, n, at, act;                 // n columns (a multiple of 4; 0: none); act: ACT_NONE for finished values
    int slices() const { return (n + kTailCols - 1) / kTailCols; }
};

template <typename XT> DEVINL void out_tail(const OutTail& t, int r, int slice, XT* x_row) {
    const int end = min(t.n, (slice + 1) * kTailCols);
    for (int j = slice * kTailCols + threadIdx.x * 4; j < end; j += blockDim.x * 4) {
        const float* p = t.in.p + (size_t)r * t.in.ld + t.col;
        float4 v;
        if (t.act == ACT_NONE) {
            v = sum_splits4(p + j, t.in.stride, t.in.splits);
        } else {
            const float4 a = sum_splits4(p + 2 * j, t.in.stride, t.in.splits), b = sum_splits4(p + 2 * j + 4, t.in.stride, t.in.splits);
            v = make_float4(glu_mul(t.act, a.x, a.y), glu_mul(t.act, a.z, a.w), glu_mul(t.act, b.x, b.y), glu_mul(t.act, b.z, b.w));
        }
        store_x4(x_row + t.at + j, v);
    }
}

// x[r, j] = o[r, j] / rms(group of j) * w[j] * act(gate[r, j]); group = 0: no norm, w = null: no weight. The values lie
// in heads of `hs` columns that start `hs_ld` apart in `o`. One CTA per row, `n` values, padded with zeros to `n_pad`.
struct GroupNormArgs {
    SplitIn o;
    int hs, hs_ld;
    int n, n_pad, group;
    const float* w;
    SplitIn gate;
    int c_gate, act;                     // act: ACT_NONE without a gate
    float eps;
};

// E consecutive values of a split input
template <int E>
DEVINL void split_load(const SplitIn& in, int row, int col, float (&v)[E]) {
    if constexpr (E == 4) {
        const float4 t = sum_splits4(in.p + (size_t)row * in.ld + col, in.stride, in.splits);
        v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
    } else {
        v[0] = in.at(row, col);
    }
}

// E: values per access; 4 when every size and column offset is a multiple of 4. grid (R, 1 + slices of the tail)
template <typename XT, int E>
__global__ void __launch_bounds__(256) group_norm_rows_kernel(const GroupNormArgs a, const OutTail tail, XT* x, int ld_x) {
    __shared__ float red[32];
    extern __shared__ __align__(16) unsigned char smem_raw[];
    float* v = reinterpret_cast<float*>(smem_raw);           // [n]
    pdl_wait();
    pdl_launch();
    const int r = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    if (blockIdx.y > 0) {
        out_tail(tail, r, blockIdx.y - 1, x + (size_t)r * ld_x);
        return;
    }
    float ss[1] = {0.0f};
    for (int j = tid * E; j < a.n; j += blockDim.x * E) {
        float t[E];
        split_load<E>(a.o, r, a.hs == a.hs_ld ? j : (j / a.hs) * a.hs_ld + j % a.hs, t);
#pragma unroll
        for (int e = 0; e < E; ++e) {
            v[j + e] = t[e];
            ss[0] += t[e] * t[e];
        }
    }
    float whole = 1.0f;
    if (a.group == a.n) {
        block_sum<1>(ss, red);
        whole = 1.0f / sqrtf(ss[0] / (float)a.n + a.eps);
    } else if (a.group > 0) {
        __syncthreads();
        for (int g = warp; g < a.n / a.group; g += 8) {
            float s = 0.0f;
            for (int j = lane; j < a.group; j += 32) s += v[g * a.group + j] * v[g * a.group + j];
            s = 1.0f / sqrtf(warp_sum(s) / (float)a.group + a.eps);
            for (int j = lane; j < a.group; j += 32) v[g * a.group + j] *= s;
        }
    }
    __syncthreads();
    for (int j = tid * E; j < a.n_pad; j += blockDim.x * E) {
        float t[E];
#pragma unroll
        for (int e = 0; e < E; ++e) t[e] = 0.0f;
        if (j < a.n) {
            if (a.act != ACT_NONE) {
                split_load<E>(a.gate, r, a.c_gate + j, t);
#pragma unroll
                for (int e = 0; e < E; ++e) t[e] = a.act == ACT_SIGMOID ? sigmoid(t[e]) : silu(t[e]);
            } else {
#pragma unroll
                for (int e = 0; e < E; ++e) t[e] = 1.0f;
            }
#pragma unroll
            for (int e = 0; e < E; ++e) {
                t[e] *= v[j + e] * whole;
                if (a.w) t[e] *= a.w[j + e];
            }
        }
        if constexpr (E == 4) {
            store_x4(x + (size_t)r * ld_x + j, make_float4(t[0], t[1], t[2], t[3]));
        } else {
            store_act(x + (size_t)r * ld_x + j, t[0]);
        }
    }
}

// ---- latent attention ---------------------------------------------------------------------------------------
// The cache row of a token is [latent (rank) | rotated key part (rot)], padded with zeros to `ld` elements; slot =
// position, pages of `page_tokens` rows. Scores and values are taken in latent space: the query is carried through
// W_uk ("absorbed") and the attention output through W_uv, so a cached token costs ld elements whatever the heads.
struct RowCache {
    void* pool;                          // [pages][kv_heads][page_tokens][ld]
    const int32_t* page_table;           // [sequences, pages_per_seq]
    int pages_per_seq, page_tokens, ld;
    int kv_heads;                        // rows of a token: 1 for latents
    DEVINL size_t row(int seq, int pos, int kvh = 0) const {
        const int page = page_table[(size_t)seq * pages_per_seq + pos / page_tokens];
        return (((size_t)page * kv_heads + kvh) * page_tokens + pos % page_tokens) * ld;
    }
};

struct LatentArgs {
    SplitIn in;                          // fused input projection
    int c_dq, c_dkv;
    int heads, dim, rot, rot_dims, vdim, rank, q_rank;
    const float *dq_norm, *dkv_norm, *inv_freq;
    float eps, scale;
    RunRows rows;
    RowCache cache;
};

// rotation of the pair (u, v) = (x[2i], x[2i+1]) at `pos`
DEVINL void rotate_pair(float& u, float& v, int pos, float inv_freq) {
    float s, c;
    sincosf((float)pos * inv_freq, &s, &c);
    const float x = u * c - v * s;
    v = v * c + u * s;
    u = x;
}

// norms the latent of row r, rotates the shared key part and stores both in the cache; whole CTA
template <typename KT>
DEVINL void latent_append(const LatentArgs& a, int r, float* red) {
    const int tid = threadIdx.x, nth = blockDim.x;
    float ss[1] = {0.0f};
    for (int j = tid; j < a.rank; j += nth) {
        const float t = a.in.at(r, a.c_dkv + j);
        ss[0] += t * t;
    }
    block_sum<1>(ss, red);
    const float s = 1.0f / sqrtf(ss[0] / (float)a.rank + a.eps);
    const int pos = a.rows.pos[r];
    KT* dst = (KT*)a.cache.pool + a.cache.row(a.rows.seq_of(r), pos);
    for (int j = tid; j < a.rank; j += nth) store_act(dst + j, a.in.at(r, a.c_dkv + j) * s * a.dkv_norm[j]);
    for (int i = tid; i < (a.rot + 1) / 2; i += nth) {
        float u = a.in.at(r, a.c_dkv + a.rank + 2 * i);
        float v = 2 * i + 1 < a.rot ? a.in.at(r, a.c_dkv + a.rank + 2 * i + 1) : 0.0f;
        if (2 * i + 1 < a.rot_dims) rotate_pair(u, v, pos, a.inv_freq[i]);
        store_act(dst + a.rank + 2 * i, u);
        if (2 * i + 1 < a.rot) store_act(dst + a.rank + 2 * i + 1, v);
    }
    for (int j = a.rank + a.rot + tid; j < a.cache.ld; j += nth) store_act(dst + j, 0.0f);
}

// many rows: x_q = normed query latent (input of W_uq, padded with zeros to ld_x), and the cache append. grid (R)
template <typename XT, typename KT>
__global__ void __launch_bounds__(256) latent_prep_kernel(const LatentArgs a, XT* x_q, int ld_x) {
    __shared__ float red[32];
    pdl_wait();
    pdl_launch();
    const int r = blockIdx.x, tid = threadIdx.x;
    float ss[1] = {0.0f};
    for (int j = tid; j < a.q_rank; j += blockDim.x) {
        const float t = a.in.at(r, a.c_dq + j);
        ss[0] += t * t;
    }
    block_sum<1>(ss, red);
    const float s = 1.0f / sqrtf(ss[0] / (float)a.q_rank + a.eps);
    for (int j = tid; j < ld_x; j += blockDim.x)
        store_act(x_q + (size_t)r * ld_x + j, j < a.q_rank ? a.in.at(r, a.c_dq + j) * s * a.dq_norm[j] : 0.0f);
    if (a.rows.tok[r] != kInactiveToken) latent_append<KT>(a, r, red);
}

// Queries in latent space, few rows: q_abs[r, h, :] = q_unrotated . W_uk[h], followed by the rotated part; f32
// [R, heads, rank + rot]. grid (heads + 1, R, slices of kLqCols latent columns); the CTAs of x == heads append the token to
// the cache when `append` is set. Two groups of threads share a column's sum. dynamic shared memory: dim + rot + 256 floats
constexpr int kLqCols = 128;
template <typename WT, typename KT>
__global__ void __launch_bounds__(256)
latent_query_kernel(const LatentArgs a, SplitIn q, const WT* w_uk, float* q_abs, int append) {
    __shared__ float red[32];
    extern __shared__ __align__(16) unsigned char smem_raw[];
    float* sq = reinterpret_cast<float*>(smem_raw);
    const int hd = blockIdx.x, r = blockIdx.y, tid = threadIdx.x;
    const int n = blockIdx.z * kLqCols + tid % kLqCols, part = tid / kLqCols;
    if (hd < a.heads)                    // this CTA's block of W_uk depends on nothing the preceding kernel writes
        for (int d = tid; d < a.dim; d += 256)
            prefetch_l2(w_uk + ((size_t)hd * a.dim + d) * a.rank + min(blockIdx.z * kLqCols, a.rank - 1));
    pdl_wait();
    pdl_launch();
    if (a.rows.tok[r] == kInactiveToken) return;
    if (hd == a.heads) {
        if (append && blockIdx.z == 0) latent_append<KT>(a, r, red);
        return;
    }
    const int dq = a.dim + a.rot;
    for (int j = tid; j < dq; j += 256) sq[j] = q.at(r, hd * dq + j);
    __syncthreads();
    float* dst = q_abs + ((size_t)r * a.heads + hd) * (a.rank + a.rot);
    float* sum = sq + dq;                // [256]
    float t = 0.0f;
    if (n < a.rank) {
        const size_t base = (size_t)hd * a.dim * a.rank + n;
        const int half = (a.dim + 1) / 2, d1 = min(a.dim, (part + 1) * half);
#pragma unroll 16
        for (int d = part * half; d < d1; ++d) t = fmaf(sq[d], WTraits<WT>::elem(w_uk, base + (size_t)d * a.rank), t);
    }
    sum[tid] = t;
    __syncthreads();
    if (part == 0 && n < a.rank) dst[n] = sum[tid] + sum[tid + kLqCols];
    if (blockIdx.z == 0) {
        const int pos = a.rows.pos[r];
        for (int i = tid; i < (a.rot + 1) / 2; i += 256) {
            float u = sq[a.dim + 2 * i], v = 2 * i + 1 < a.rot ? sq[a.dim + 2 * i + 1] : 0.0f;
            if (2 * i + 1 < a.rot_dims) rotate_pair(u, v, pos, a.inv_freq[i]);
            dst[a.rank + 2 * i] = u;
            if (2 * i + 1 < a.rot) dst[a.rank + 2 * i + 1] = v;
        }
    }
}

// many rows: the unrotated query parts as BF16 operands of the per-head products with W_uk^T, [heads][R][ld_u], and the
// rotated parts in f32, [R, heads, rot]. grid (R)
__global__ void __launch_bounds__(256)
latent_split_query_kernel(const LatentArgs a, int R, SplitIn q, uint16_t* x_u, int ld_u, float* q_rot) {
    pdl_wait();
    pdl_launch();
    const int r = blockIdx.x, dq = a.dim + a.rot, pos = a.rows.pos[r];
    for (int j = threadIdx.x; j < a.heads * ld_u; j += blockDim.x) {
        const int hd = j / ld_u, d = j % ld_u;
        store_act(x_u + ((size_t)hd * R + r) * ld_u + d, d < a.dim ? q.at(r, hd * dq + d) : 0.0f);
    }
    const int half = (a.rot + 1) / 2;
    for (int j = threadIdx.x; j < a.heads * half; j += blockDim.x) {
        const int hd = j / half, i = j % half, c = hd * dq + a.dim + 2 * i;
        float u = q.at(r, c), v = 2 * i + 1 < a.rot ? q.at(r, c + 1) : 0.0f;
        if (2 * i + 1 < a.rot_dims) rotate_pair(u, v, pos, a.inv_freq[i]);
        float* dst = q_rot + ((size_t)r * a.heads + hd) * a.rot + 2 * i;
        dst[0] = u;
        if (2 * i + 1 < a.rot) dst[1] = v;
    }
}

// Split-KV partials of attention, `rank` value columns: `o` un-normalised [splits][R * heads][rank], `ml` (running maximum,
// denominator) [splits][R * heads][2]; a split without a visible key has denominator 0 and leaves `o` unwritten.
struct AttnPart {
    float* o;
    float* ml;
    int splits;
    size_t rows;                         // R * heads
};

// Attention of one (row, head, split) per CTA on the CUDA cores: f32 caches, BF16 weights with an f32 cache, and heads
// too wide for the tensor-core kernels. The key of a cache row is its first `dk` elements; its value is `vw` elements
// from `v_at` on (latent attention: from 0 on, RPL registers hold them for both). Query heads share the cache rows of
// kv head (head / group). Queries [R, heads, dk] f32. grid (heads, R, splits), 256 threads, dynamic shared memory
// dk + 8 * vw + 16 floats. vw <= 32 * RPL.
struct RowAttnArgs {
    const float* q;
    int heads, group, dk, v_at, vw;
    float scale;
    RunRows rows;
    RowCache cache;
    AttnPart part;
};

template <typename KT, int RPL, bool LATENT>
__global__ void __launch_bounds__(256) row_attn_kernel(const RowAttnArgs a) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const AttnPart& part = a.part;
    const int DK = a.dk, VW = a.vw;
    float* sq = reinterpret_cast<float*>(smem_raw);          // [DK]
    float* so = sq + DK;                                     // [8][VW]
    float* sm = so + 8 * VW;                                 // [8][2]
    pdl_wait();
    pdl_launch();
    const int hd = blockIdx.x, r = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const size_t pr = (size_t)blockIdx.z * part.rows + (size_t)r * a.heads + hd;
    if (a.rows.tok[r] == kInactiveToken) return;
    const int visible = a.rows.pos[r] + 1, seq = a.rows.seq_of(r);
    const int per = (visible + part.splits - 1) / part.splits;
    const int p0 = blockIdx.z * per, p1 = min(visible, p0 + per);
    if (p0 >= p1) {
        if (tid == 0) { part.ml[2 * pr] = -INFINITY; part.ml[2 * pr + 1] = 0.0f; }
        return;
    }
    const float* q = a.q + ((size_t)r * a.heads + hd) * DK;
    for (int j = tid; j < DK; j += 256) sq[j] = q[j];
    __syncthreads();
    const int kvh = hd / a.group;
    float m = -INFINITY, l = 0.0f, acc[RPL];
#pragma unroll
    for (int i = 0; i < RPL; ++i) acc[i] = 0.0f;
    for (int p = p0 + warp; p < p1; p += 8) {
        const KT* row = (const KT*)a.cache.pool + a.cache.row(seq, p, kvh);
        float c[RPL], s = 0.0f;
#pragma unroll
        for (int i = 0; i < RPL; ++i) {
            const int j = lane + 32 * i;
            c[i] = j < VW ? WTraits<KT>::elem(row, (LATENT ? 0 : a.v_at) + j) : 0.0f;
            if (LATENT && j < VW) s = fmaf(sq[j], c[i], s);
        }
        for (int j = (LATENT ? VW : 0) + lane; j < DK; j += 32) s = fmaf(sq[j], WTraits<KT>::elem(row, j), s);
        s = warp_sum(s) * a.scale;
        const float m2 = fmaxf(m, s), f = expf(m - m2), e = expf(s - m2);
        l = l * f + e;
#pragma unroll
        for (int i = 0; i < RPL; ++i) acc[i] = fmaf(e, c[i], acc[i] * f);
        m = m2;
    }
#pragma unroll
    for (int i = 0; i < RPL; ++i)
        if (lane + 32 * i < VW) so[warp * VW + lane + 32 * i] = acc[i];
    if (lane == 0) { sm[2 * warp] = m; sm[2 * warp + 1] = l; }
    __syncthreads();
    float M = -INFINITY, L = 0.0f;
    for (int w = 0; w < 8; ++w) M = fmaxf(M, sm[2 * w]);
    for (int w = 0; w < 8; ++w) L += sm[2 * w + 1] > 0.0f ? sm[2 * w + 1] * expf(sm[2 * w] - M) : 0.0f;
    for (int j = tid; j < VW; j += 256) {
        float t = 0.0f;
        for (int w = 0; w < 8; ++w)
            if (sm[2 * w + 1] > 0.0f) t += so[w * VW + j] * expf(sm[2 * w] - M);
        part.o[pr * VW + j] = t;
    }
    if (tid == 0) { part.ml[2 * pr] = M; part.ml[2 * pr + 1] = L; }
}

// attention output of (row, head): column j of `rank`, partials added in split order; `sc` [splits] holds the factors
// exp(m_s - M) / L of attn_part_factors. `sink`: score of one more term of the denominator that has no value, or null.
DEVINL void attn_part_factors(const AttnPart& part, size_t rh, float* sc, const float* sink = nullptr) {
    if (threadIdx.x < 32) {
        float M = sink ? *sink : -INFINITY;
        for (int s = threadIdx.x; s < part.splits; s += 32) {
            const float* ml = part.ml + 2 * ((size_t)s * part.rows + rh);
            if (__ldcg(ml + 1) > 0.0f) M = fmaxf(M, __ldcg(ml));
        }
        M = warp_max(M);
        float L = 0.0f;
        for (int s = threadIdx.x; s < part.splits; s += 32) {
            const float* ml = part.ml + 2 * ((size_t)s * part.rows + rh);
            const float l = __ldcg(ml + 1), f = l > 0.0f ? expf(__ldcg(ml) - M) : 0.0f;
            sc[s] = f;
            L += l * f;
        }
        L = warp_sum(L);
        if (sink) L += expf(*sink - M);
        __syncwarp();
        for (int s = threadIdx.x; s < part.splits; s += 32) sc[s] = L > 0.0f ? sc[s] / L : 0.0f;
    }
    __syncthreads();
}
DEVINL float attn_part_value(const AttnPart& part, size_t rh, int rank, int j, const float* sc) {
    const float* o = part.o + rh * rank + j;
    const size_t stride = part.rows * rank;
    float t = 0.0f;
    for (int s0 = 0; s0 < part.splits; s0 += 8) {
        float v[8];
#pragma unroll
        for (int q = 0; q < 8; ++q) v[q] = s0 + q < part.splits && sc[s0 + q] > 0.0f ? __ldcg(o + (s0 + q) * stride) : 0.0f;
#pragma unroll
        for (int q = 0; q < 8; ++q)
            if (s0 + q < part.splits) t = fmaf(v[q], sc[s0 + q], t);
    }
    return t;
}

// many rows: merged output as BF16 operands of the per-head products with W_uv, [heads][R][ld]. grid (heads, R)
__global__ void __launch_bounds__(128)
latent_merge_kernel(int R, int heads, int rank, AttnPart part, uint16_t* x, int ld) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    float* sc = reinterpret_cast<float*>(smem_raw);
    pdl_wait();
    pdl_launch();
    const int hd = blockIdx.x, r = blockIdx.y;
    const size_t rh = (size_t)r * heads + hd;
    attn_part_factors(part, rh, sc);
    for (int j = threadIdx.x; j < ld; j += 128)
        store_act(x + ((size_t)hd * R + r) * ld + j, j < rank ? attn_part_value(part, rh, rank, j, sc) : 0.0f);
}

// few rows: merge, W_uv and the output gate: out[r, h * vdim + v] = (W_uv[h, v, :] . o) * sigmoid(gate). W_uv rows are
// `ldw` elements apart. A warp owns four value columns; rows of whole 16-byte pieces are fetched before the dependency wait.
// grid (heads, R, slices of 32 value columns), 256 threads, shared memory splits + rank floats (16-byte aligned)
template <typename WT>
__global__ void __launch_bounds__(256)
latent_out_kernel(int heads, int rank, int vdim, AttnPart part, const WT* w_uv, int ldw, SplitIn gate, int c_gate,
                  const uint32_t* tok, float* out, int ld_out) {
    constexpr int EPL = WTraits<WT>::EPL, PIECES = 512 / (32 * EPL);         // rank <= 512
    extern __shared__ __align__(16) unsigned char smem_raw[];
    float* so = reinterpret_cast<float*>(smem_raw);
    float* sc = so + (rank + 3) / 4 * 4;
    const int hd = blockIdx.x, r = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int vb = blockIdx.z * 32 + warp * 4;
    const bool vec = rank % EPL == 0 && ldw % EPL == 0;
    uint4 w[4][PIECES];
    if (vec) {
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int p = 0; p < PIECES; ++p) {
                const int j = (p * 32 + lane) * EPL;
                w[i][p] = make_uint4(0u, 0u, 0u, 0u);
                if (vb + i < vdim && j < rank) w[i][p] = ldg_stream16(w_uv + ((size_t)hd * vdim + vb + i) * ldw + j);
            }
    }
    pdl_wait();
    pdl_launch();
    if (tok[r] == kInactiveToken) return;
    const size_t rh = (size_t)r * heads + hd;
    attn_part_factors(part, rh, sc);
    for (int j = threadIdx.x; j < rank; j += 256) so[j] = attn_part_value(part, rh, rank, j, sc);
    __syncthreads();
    float t[4] = {0.0f, 0.0f, 0.0f, 0.0f};
    if (vec) {
#pragma unroll
        for (int p = 0; p < PIECES; ++p) {
            const int j = (p * 32 + lane) * EPL;
            if (j < rank)
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int e = 0; e < EPL; ++e) t[i] = fmaf(WTraits<WT>::elem(&w[i][p], e), so[j + e], t[i]);
        }
    } else {
        for (int i = 0; i < 4 && vb + i < vdim; ++i)
            for (int j = lane; j < rank; j += 32) t[i] = fmaf(WTraits<WT>::elem(w_uv, ((size_t)hd * vdim + vb + i) * ldw + j), so[j], t[i]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        t[i] = warp_sum(t[i]);
        if (lane == 0 && vb + i < vdim) {
            const int c = hd * vdim + vb + i;
            out[(size_t)r * ld_out + c] = t[i] * sigmoid(gate.at(r, c_gate + c));
        }
    }
}

// ---- grouped-query attention with whole-projection norms ------------------------------------------------------
// The cache row of a (token, kv head) is [key, zero-padded to kd | value, zero-padded], no ring: slot = position. q and k
// get their biases, are divided by the root mean square over all heads together and weighted; q is also multiplied by
// 1 + coef * ln(floor((p + 1) / every) + 1).
struct HeadAttnArgs {
    SplitIn in;                          // fused input projection
    int c_q, c_k, c_v;
    int heads, kv_heads, dim, vdim, kd;
    const float *q_b, *k_b, *v_b, *q_norm, *k_norm;
    float eps, temp_coef;
    int temp_every;
    RunRows rows;
    RowCache cache;
};

template <int E> DEVINL void store_act_e(uint16_t* p, const float (&v)[E]) {
    if constexpr (E == 4) store_x4(p, make_float4(v[0], v[1], v[2], v[3]));
    else store_act(p, v[0]);
}
template <int E> DEVINL void store_act_e(float* p, const float (&v)[E]) {
    if constexpr (E == 4) store_x4(p, make_float4(v[0], v[1], v[2], v[3]));
    else store_act(p, v[0]);
}

// Queries [R, heads, ld_q] (BF16 rows padded with zeros for the tensor-core kernel, f32 rows of dim values for the other one)
// and the cache append. E: values per access, 4 when the head sizes are multiples of 4. grid (R, 3): queries, keys, values;
// up to 1024 threads. dynamic shared memory heads * dim floats.
template <typename QT, typename KT, int E>
__global__ void __launch_bounds__(1024) head_prep_kernel(const HeadAttnArgs a, QT* q_out, int ld_q) {
    __shared__ float red[32];
    extern __shared__ __align__(16) unsigned char smem_raw[];
    float* v = reinterpret_cast<float*>(smem_raw);
    pdl_wait();
    pdl_launch();
    const int r = blockIdx.x, part = blockIdx.y, tid = threadIdx.x;
    if (a.rows.tok[r] == kInactiveToken) return;
    const int pos = a.rows.pos[r], seq = a.rows.seq_of(r);
    KT* pool = (KT*)a.cache.pool;
    float t[E];
    if (part == 2) {
        const int vp = a.cache.ld - a.kd;
        for (int i = tid * E; i < a.kv_heads * vp; i += blockDim.x * E) {
            const int g = i / vp, d = i % vp, c = g * a.vdim + d;
#pragma unroll
            for (int e = 0; e < E; ++e) t[e] = 0.0f;
            if (d < a.vdim) {
                split_load<E>(a.in, r, a.c_v + c, t);
#pragma unroll
                for (int e = 0; e < E; ++e) t[e] += a.v_b[c + e];
            }
            store_act_e<E>(pool + a.cache.row(seq, pos, g) + a.kd + d, t);
        }
        return;
    }
    const bool key = part == 1;
    const int n = (key ? a.kv_heads : a.heads) * a.dim, col = key ? a.c_k : a.c_q;
    const float *bias = key ? a.k_b : a.q_b, *w = key ? a.k_norm : a.q_norm;
    float ss[1] = {0.0f};
    for (int i = tid * E; i < n; i += blockDim.x * E) {
        split_load<E>(a.in, r, col + i, t);
#pragma unroll
        for (int e = 0; e < E; ++e) {
            t[e] += bias[i + e];
            v[i + e] = t[e];
            ss[0] += t[e] * t[e];
        }
    }
    block_sum<1>(ss, red);
    float s = 1.0f / sqrtf(ss[0] / (float)n + a.eps);
    if (!key) s *= 1.0f + a.temp_coef * logf((float)((pos + 1) / a.temp_every) + 1.0f);
    const int ld = key ? a.kd : ld_q, heads = key ? a.kv_heads : a.heads;
    for (int i = tid * E; i < heads * ld; i += blockDim.x * E) {
        const int h = i / ld, d = i % ld, c = h * a.dim + d;
#pragma unroll
        for (int e = 0; e < E; ++e) t[e] = d < a.dim ? v[c + e] * s * w[c + e] : 0.0f;
        if (key) store_act_e<E>(pool + a.cache.row(seq, pos, h) + d, t);
        else store_act_e<E>(q_out + ((size_t)r * a.heads + h) * ld_q + d, t);
    }
}

// Merge of the split partials, with the sink, into the output projection's input; grid (heads + slices of the tail, R),
// dynamic shared memory: splits floats
template <typename XT>
__global__ void __launch_bounds__(128)
head_merge_kernel(int heads, int vdim, AttnPart part, const float* sink, const OutTail tail, XT* x, int ld_x) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    float* sc = reinterpret_cast<float*>(smem_raw);
    pdl_wait();
    pdl_launch();
    const int hd = blockIdx.x, r = blockIdx.y;
    if (hd >= heads) {
        out_tail(tail, r, hd - heads, x + (size_t)r * ld_x);
        return;
    }
    const size_t rh = (size_t)r * heads + hd;
    attn_part_factors(part, rh, sc, sink + hd);
    for (int j = threadIdx.x; j < vdim; j += 128) store_act(x + (size_t)r * ld_x + hd * vdim + j, attn_part_value(part, rh, vdim, j, sc));
}

}  // namespace oxg4
