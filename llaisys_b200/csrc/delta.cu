// Gated delta rule with a decay per key channel: a recurrent mixer whose memory per head is a matrix S [key channels,
// value channels] in float32 that every token decays, corrects towards its value and reads:
//
//     S <- diag(g_t) S,   u_t = beta_t (v_t - S^T k_t),   S <- S + k_t u_t^T,   o_t = S^T q_t
//
// q and k have G heads, v, g and beta H heads (a multiple of G); value head h works with query/key head h / (H / G).
//
//  * delta_prep        what enters the recurrence, from the projections: a short causal convolution per channel and silu on
//                      q, k and v; q and k made unit vectors per head (q then scaled); the decays
//                      g = exp(-exp(A_h) softplus(z)); beta = sigmoid(b).  A warp per token and head.  The convolution's
//                      last taps - 1 inputs are carried from step to step in a state row per sequence.
//  * delta_scan        the recurrence token by token in float32: short steps, single tokens, and the 32-bit path.
//  * delta_chunk and delta_walk    long steps in chunks of 16 tokens.  With G_t the product of the decays from the chunk's
//                      start to token t and S_0 the state at its start, the corrections of a chunk are
//                          u = T (V - (K . G) S_0),   T = (I + diag(beta) A)^-1 diag(beta),
//                          A_ts = sum_i k_t[i] k_s[i] g_(s+1)[i] .. g_t[i]   for s < t,
//                      and with B_ts the same sums with q_t in k_t's place (s <= t) the results are
//                          o = (Q . G) S_0 + B u = (Q . G - B T (K . G)) S_0 + B T V.
//                      So all that does not contain S_0 is computed for every chunk side by side (delta_chunk), and only three
//                      matrix products with the state a chunk remain sequential (delta_walk).  Decays are only ever multiplied up, never divided, so a channel that
//                      forgets at once costs nothing but its products.
//                      delta_walk runs on the tensor cores: four warps share 16 value columns of S as accumulator fragments,
//                      which are the A operand of the next chunk's products without leaving the registers.  Every float32 operand
//                      is split in two TF32 numbers (hi + lo) and a product is hi hi + hi lo + lo hi, which keeps
//                      about 21 bits of each factor; sums are float32.
#include "common.cuh"

namespace {

constexpr float UNIT_EPS = 1e-6f;       // inside the root of the unit vectors

struct DeltaPrepParams {
    const float* proj;        // [T, ld]: q (G dk), k (G dk), v (H dv), b (H), before the convolution
    int ld;
    float* z;                 // [T, H dk]: the decays' logits, replaced by the decays
    const float* conv_w;      // [taps, C], C = 2 G dk + H dv (taps - 1: the current token's)
    const float* a_log;       // [H]
    float* conv_state;        // [slots, (taps - 1) * C], oldest input first
    const int* seq_start;     // [B + 1]
    const int* seq_slot;      // [B]
    float* out;               // [T, C]
    float* beta;              // [T, H]
    int G, H, dk, dv, taps;
    float q_scale;
    int fast;                 // the bfloat16 path: the activation by the special-function unit
    int vec;                  // (set by the entry point) rows of 16-byte pieces
};

__device__ __forceinline__ float silu(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

constexpr int PREP_WARPS = 4;
constexpr int PREP_TOKENS = 8;          // consecutive tokens of a sequence that a warp takes, or as many as the convolution
                                        // reaches back: only a sequence's first run reads the carried inputs
__host__ __device__ constexpr int prep_run(int taps) { return taps - 1 > PREP_TOKENS ? taps - 1 : PREP_TOKENS; }

// N float32 values from / to an address aligned to N * 4 bytes.
template <int N> __device__ __forceinline__ void load_vec(float (&v)[N], const float* src) {
    if constexpr (N == 4) { const float4 x = *reinterpret_cast<const float4*>(src); v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w; }
    else if constexpr (N == 2) { const float2 x = *reinterpret_cast<const float2*>(src); v[0] = x.x; v[1] = x.y; }
    else { for (int e = 0; e < N; ++e) v[e] = src[e]; }
}
template <int N> __device__ __forceinline__ void store_vec(float* dst, const float (&v)[N]) {
    if constexpr (N == 4) *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]);
    else if constexpr (N == 2) *reinterpret_cast<float2*>(dst) = make_float2(v[0], v[1]);
    else { for (int e = 0; e < N; ++e) dst[e] = v[e]; }
}

// A warp per run of tokens and unit: a q, k or v head (convolution, silu, unit vector), or a head's decays and step sizes.
// PER channels a lane: neighbours in one access (VEC: heads of 32 PER channels, aligned rows) or 32 apart.  TAPS > 0: that
// many taps, the inputs of the run in registers; 0: any number, every input read where it is needed.  FAST: silu by the
// special-function unit.  The warp of a sequence's first run is the only one that reads the carried inputs, and it leaves the
// new ones (which depend on them and on the step's own inputs only).
template <int TAPS, int PER, bool VEC, bool FAST>
__device__ __forceinline__ void prep_head(const DeltaPrepParams& p, int unit, int b, int tok0, int n, int at0, int lane) {
    const int C = 2 * p.G * p.dk + p.H * p.dv, taps = TAPS > 0 ? TAPS : p.taps, back = taps - 1;
    const bool is_qk = unit < 2 * p.G;
    const int d = is_qk ? p.dk : p.dv;
    const int c0 = (is_qk ? unit * p.dk : 2 * p.G * p.dk + (unit - 2 * p.G) * p.dv) + (VEC ? lane * PER : lane);
    const float mult = unit < p.G ? p.q_scale : 1.f;
    float* st = p.conv_state + (size_t)p.seq_slot[b] * back * C + c0;      // [back][C]
    const float* x = p.proj + (size_t)tok0 * p.ld + c0;                    // input of the sequence's token r: x + r * ld
    float* out = p.out + (size_t)tok0 * C + c0;
    const int hi = min(n, at0 + prep_run(taps));
    auto have = [&](int e) { return VEC || lane + e * 32 < d; };
    auto load = [&](float (&v)[PER], const float* src) {
        if constexpr (VEC) load_vec<PER>(v, src);
        else {
#pragma unroll
            for (int e = 0; e < PER; ++e) v[e] = have(e) ? src[e * 32] : 0.f;
        }
    };
    auto store = [&](float* dst, const float (&v)[PER]) {
        if constexpr (VEC) store_vec<PER>(dst, v);
        else {
#pragma unroll
            for (int e = 0; e < PER; ++e)
                if (have(e)) dst[e * 32] = v[e];
        }
    };
    auto finish = [&](int t, float (&v)[PER]) {
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < PER; ++e) {
            v[e] = FAST ? __fdividef(v[e], 1.0f + __expf(-v[e])) : silu(v[e]);
            ss = fmaf(v[e], v[e], ss);
        }
        if (is_qk) {
            const float f = mult / sqrtf(warp_sum(ss) + UNIT_EPS);
#pragma unroll
            for (int e = 0; e < PER; ++e) v[e] *= f;
        }
        store(out + (size_t)t * C, v);
    };
    if constexpr (TAPS > 0) {
        constexpr int BACK = TAPS - 1;
        float w[TAPS][PER], in[BACK + PREP_TOKENS][PER];
#pragma unroll
        for (int j = 0; j < BACK + PREP_TOKENS; ++j) {
            const int r = at0 - BACK + j;
#pragma unroll
            for (int e = 0; e < PER; ++e) in[j][e] = 0.f;
            if (r < hi) load(in[j], r >= 0 ? x + (ptrdiff_t)r * p.ld : st + (size_t)(r + BACK) * C);
        }
#pragma unroll
        for (int j = 0; j < TAPS; ++j) load(w[j], p.conv_w + (size_t)j * C + c0);
#pragma unroll
        for (int u = 0; u < PREP_TOKENS; ++u) {
            if (at0 + u >= hi) break;                                      // (uniform)
            float v[PER];
#pragma unroll
            for (int e = 0; e < PER; ++e) {
                v[e] = 0.f;
#pragma unroll
                for (int j = 0; j < TAPS; ++j) v[e] = fmaf(w[j][e], in[u + j][e], v[e]);
            }
            finish(at0 + u, v);
        }
        if (at0 == 0) {
#pragma unroll
            for (int j = 0; j < BACK; ++j) {                               // the input of token n - BACK + j
                float v[PER];
                if (n - BACK + j >= PREP_TOKENS) {
                    load(v, x + (ptrdiff_t)(n - BACK + j) * p.ld);
                } else {
#pragma unroll
                    for (int e = 0; e < PER; ++e) v[e] = 0.f;
#pragma unroll
                    for (int k = 0; k < BACK + PREP_TOKENS; ++k)
                        if (k == n + j) {
#pragma unroll
                            for (int e = 0; e < PER; ++e) v[e] = in[k][e];
                        }
                }
                store(st + (size_t)j * C, v);
            }
        }
    } else {
        for (int t = at0; t < hi; ++t) {
            float v[PER];
#pragma unroll
            for (int e = 0; e < PER; ++e) v[e] = 0.f;
            for (int j = 0; j < taps; ++j) {
                const int r = t - back + j;
                float in[PER], w[PER];
                load(in, r >= 0 ? x + (ptrdiff_t)r * p.ld : st + (size_t)(r + back) * C);
                load(w, p.conv_w + (size_t)j * C + c0);
#pragma unroll
                for (int e = 0; e < PER; ++e) v[e] = fmaf(w[e], in[e], v[e]);
            }
            finish(t, v);
        }
        if (at0 == 0)
            for (int j = 0; j < back; ++j) {                               // ascending: what is still needed is not overwritten
                const int r = n - back + j;
                float v[PER];
                load(v, r >= 0 ? x + (ptrdiff_t)r * p.ld : st + (size_t)(j + n) * C);
                store(st + (size_t)j * C, v);
            }
    }
}

template <int TAPS, bool FAST>
__global__ void __launch_bounds__(PREP_WARPS * 32, 6) delta_prep_kernel(DeltaPrepParams p) {
    const int lane = threadIdx.x & 31, unit = blockIdx.y, b = blockIdx.z;
    const int run = TAPS > 0 ? prep_run(TAPS) : prep_run(p.taps);
    const int at0 = (blockIdx.x * PREP_WARPS + (threadIdx.x >> 5)) * run;
    const int tok0 = p.seq_start[b], n = p.seq_start[b + 1] - tok0;
    llb_grid_dependency_sync();
    if (at0 >= n) return;
    if (unit >= 2 * p.G + p.H) {                           // a head's decays and its step sizes
        const int h = unit - 2 * p.G - p.H, C = 2 * p.G * p.dk + p.H * p.dv;
        const float rate = expf(p.a_log[h]);
        const size_t step = (size_t)p.H * p.dk;
        for (int t0 = at0; t0 < min(n, at0 + run); t0 += PREP_TOKENS) {
            const int m = min(min(n, at0 + run) - t0, PREP_TOKENS);
            float* z = p.z + ((size_t)(tok0 + t0) * p.H + h) * p.dk;
            if (lane < m) {
                const size_t t = (size_t)(tok0 + t0 + lane);
                p.beta[t * p.H + h] = 1.0f / (1.0f + expf(-p.proj[t * p.ld + C + h]));
            }
            for (int i = lane; i < p.dk; i += 32) {
                float v[PREP_TOKENS];
#pragma unroll
                for (int u = 0; u < PREP_TOKENS; ++u) v[u] = u < m ? z[u * step + i] : 0.f;
#pragma unroll
                for (int u = 0; u < PREP_TOKENS; ++u)
                    if (u < m) z[u * step + i] = expf(-rate * softplus(v[u]));
            }
        }
        return;
    }
    const int d = unit < 2 * p.G ? p.dk : p.dv;
    if (d == 128 && p.vec) prep_head<TAPS, 4, true, FAST>(p, unit, b, tok0, n, at0, lane);
    else if (d == 64 && p.vec) prep_head<TAPS, 2, true, FAST>(p, unit, b, tok0, n, at0, lane);
    else if (d <= 32) prep_head<TAPS, 1, false, FAST>(p, unit, b, tok0, n, at0, lane);
    else if (d <= 64) prep_head<TAPS, 2, false, FAST>(p, unit, b, tok0, n, at0, lane);
    else if (d <= 128) prep_head<TAPS, 4, false, FAST>(p, unit, b, tok0, n, at0, lane);
    else prep_head<0, 8, false, FAST>(p, unit, b, tok0, n, at0, lane);
}

// ------------------------------------------------------------------ the recurrence, token by token
struct DeltaScanParams {
    const float* qkv;         // [T, C]: q (G dk), k (G dk), v (H dv)
    const float* g;           // [T, H dk]
    const float* beta;        // [T, H]
    float* state;             // [slots, H dk dv]
    const int* seq_start;     // [B + 1]
    const int* seq_slot;      // [B]
    float* out;               // [T, H dv]
    int G, H, dk, dv;
};

constexpr int SCAN_THREADS = 128;
constexpr int SCAN_STAGE = 16;          // tokens staged in shared memory at a time
constexpr int SCAN_GROUP = 4;           // tokens whose read-outs are reduced together
constexpr int scan_pad(int kpt) { return (kpt / 4) % 2 == 1 ? 0 : 4; }

// KS lanes share a value column, each with KPT consecutive key channels (a multiple of 4); a block of 128 threads owns
// 128 / KS columns of one head of one sequence.  In shared memory the lanes' groups of a token's k, q and g lie an odd
// number of 16-byte pieces apart, so that the 16-byte reads of a quarter-warp fall on different banks.
template <int KS, int KPT>
__global__ void __launch_bounds__(SCAN_THREADS) delta_scan_kernel(DeltaScanParams p) {
    extern __shared__ __align__(16) float sm[];
    constexpr int COLS = SCAN_THREADS / KS, DKP = KS * KPT, PAD = scan_pad(KPT), ROW = KS * (KPT + PAD);
    float* sq = sm;
    float* sk = sq + SCAN_STAGE * ROW;
    float* sg = sk + SCAN_STAGE * ROW;
    float* sv = sg + SCAN_STAGE * ROW;                     // [STAGE][COLS]
    float* sb = sv + SCAN_STAGE * COLS;                    // [STAGE]
    const int tid = threadIdx.x, part = tid & (KS - 1), cloc = tid / KS;
    const int col = blockIdx.x * COLS + cloc, h = blockIdx.y, b = blockIdx.z;
    const int dk = p.dk, dv = p.dv, kh = h / (p.H / p.G), C = 2 * p.G * dk + p.H * dv;
    llb_grid_dependency_sync();
    const int tok0 = p.seq_start[b], n = p.seq_start[b + 1] - tok0;
    float* st = p.state + ((size_t)p.seq_slot[b] * p.H + h) * dk * dv;
    float S[KPT];
#pragma unroll
    for (int m = 0; m < KPT; ++m) {
        const int i = part * KPT + m;
        S[m] = (i < dk && col < dv) ? st[(size_t)i * dv + col] : 0.f;
    }
    for (int c0 = 0; c0 < n; c0 += SCAN_STAGE) {
        const int nc = min(SCAN_STAGE, n - c0), ng = (nc + SCAN_GROUP - 1) / SCAN_GROUP * SCAN_GROUP;
        __syncthreads();
        // (places past the step's end hold g = 1, k = q = 0, beta = 0: they leave the state as it is)
        for (int idx = tid; idx < ng * DKP; idx += SCAN_THREADS) {
            const int t = idx / DKP, i = idx - t * DKP, w = t * ROW + (i / KPT) * (KPT + PAD) + (i % KPT);
            const bool in = t < nc && i < dk;
            const size_t row = (size_t)(tok0 + c0 + t);
            sq[w] = in ? p.qkv[row * C + kh * dk + i] : 0.f;
            sk[w] = in ? p.qkv[row * C + (p.G + kh) * dk + i] : 0.f;
            sg[w] = in ? p.g[(row * p.H + h) * dk + i] : 1.f;
        }
        for (int idx = tid; idx < ng * COLS; idx += SCAN_THREADS) {
            const int t = idx / COLS, cc = blockIdx.x * COLS + idx - t * COLS;
            sv[idx] = (t < nc && cc < dv) ? p.qkv[(size_t)(tok0 + c0 + t) * C + 2 * p.G * dk + h * dv + cc] : 0.f;
        }
        if (tid < ng) sb[tid] = tid < nc ? p.beta[(size_t)(tok0 + c0 + tid) * p.H + h] : 0.f;
        __syncthreads();
        for (int t0 = 0; t0 < nc; t0 += SCAN_GROUP) {
            float acc[SCAN_GROUP];
#pragma unroll
            for (int u = 0; u < SCAN_GROUP; ++u) {
                const int t = t0 + u, w = t * ROW + part * (KPT + PAD);
                const float4* g4 = reinterpret_cast<const float4*>(sg + w);
                const float4* k4 = reinterpret_cast<const float4*>(sk + w);
                const float4* q4 = reinterpret_cast<const float4*>(sq + w);
                float r[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                for (int m = 0; m < KPT; m += 4) {
                    const float4 g = g4[m / 4], k = k4[m / 4];
                    S[m] *= g.x;
                    S[m + 1] *= g.y;
                    S[m + 2] *= g.z;
                    S[m + 3] *= g.w;
                    r[0] = fmaf(S[m], k.x, r[0]);
                    r[1] = fmaf(S[m + 1], k.y, r[1]);
                    r[2] = fmaf(S[m + 2], k.z, r[2]);
                    r[3] = fmaf(S[m + 3], k.w, r[3]);
                }
                float read = (r[0] + r[1]) + (r[2] + r[3]);
#pragma unroll
                for (int o = 1; o < KS; o <<= 1) read += __shfl_xor_sync(0xffffffffu, read, o);
                const float upd = sb[t] * (sv[t * COLS + cloc] - read);
                float o4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                for (int m = 0; m < KPT; m += 4) {
                    const float4 k = k4[m / 4], q = q4[m / 4];
                    S[m] = fmaf(k.x, upd, S[m]);
                    S[m + 1] = fmaf(k.y, upd, S[m + 1]);
                    S[m + 2] = fmaf(k.z, upd, S[m + 2]);
                    S[m + 3] = fmaf(k.w, upd, S[m + 3]);
                    o4[0] = fmaf(S[m], q.x, o4[0]);
                    o4[1] = fmaf(S[m + 1], q.y, o4[1]);
                    o4[2] = fmaf(S[m + 2], q.z, o4[2]);
                    o4[3] = fmaf(S[m + 3], q.w, o4[3]);
                }
                acc[u] = (o4[0] + o4[1]) + (o4[2] + o4[3]);
            }
#pragma unroll
            for (int o = 1; o < KS; o <<= 1) {
#pragma unroll
                for (int u = 0; u < SCAN_GROUP; ++u) acc[u] += __shfl_xor_sync(0xffffffffu, acc[u], o);
            }
            if (part == 0 && col < dv) {
#pragma unroll
                for (int u = 0; u < SCAN_GROUP; ++u)
                    if (t0 + u < nc) p.out[(size_t)(tok0 + c0 + t0 + u) * p.H * dv + h * dv + col] = acc[u];
            }
        }
    }
#pragma unroll
    for (int m = 0; m < KPT; ++m) {
        const int i = part * KPT + m;
        if (i < dk && col < dv) st[(size_t)i * dv + col] = S[m];
    }
}

// ------------------------------------------------------------------ long steps, chunk by chunk
constexpr int CHUNK = 16;
constexpr int CHUNK_THREADS = 128;

struct DeltaChunkParams {
    const float* qkv;
    const float* g;
    const float* beta;
    float* state;
    const int* seq_start;
    const int* seq_slot;
    float* out;
    float* rec;               // [chunks, H, rec_floats]
    int* err;                 // set when a bounded wait runs out
    int G, H, dk, dv;
    int cb;                   // blocks of 16 value columns
};

// What delta_chunk leaves for one chunk of one head, in floats, with np blocks of 16 key channels.  W, Q and K are stored as
// the fragments that delta_walk multiplies with: 16-byte pieces, lane by lane.
__host__ __device__ constexpr int rec_q(int np) { return 256 * np; }           // (W stands at 0)
__host__ __device__ constexpr int rec_k(int np) { return 512 * np; }
__host__ __device__ constexpr int rec_gam(int np) { return 768 * np; }
__host__ __device__ constexpr int rec_u(int np) { return 784 * np; }           // per block of value columns: 256 of T V, 256 of B T V
__host__ __device__ constexpr int rec_floats(int np, int cb) { return rec_u(np) + 512 * cb; }

// The first chunk's place among all chunks of the step: sequences need not start at multiples of 16, and two never collide.
__device__ __forceinline__ int chunk_base(int tok0, int b) { return tok0 / CHUNK + b; }

// Fragment order.  A tile of 8 columns of the chunk's tokens holds the tokens 4 (n / 2) + n % 2 + 2 tile, n = 0 .. 7, and a
// tile of 8 key channels of block p the channels 16 p + 4 (n / 2) + n % 2 + 2 half: so the two TF32 steps of a pair of tiles
// find their operands in one 16-byte piece.
__device__ __forceinline__ int frag_index(int n, int tile) { return 4 * (n >> 1) + (n & 1) + 2 * tile; }

// NPK: blocks of 16 key channels per warp of delta_walk (four warps share a head's channels).
template <int NPK>
__global__ void __launch_bounds__(CHUNK_THREADS, 5) delta_chunk_kernel(DeltaChunkParams p) {
    extern __shared__ __align__(16) float sm[];
    constexpr int NP = 4 * NPK, DKP = 16 * NP, LD = DKP + 4;      // rows 16-byte aligned; a step of 4 banks from row to row
    const int b = blockIdx.z, h = blockIdx.y, c = blockIdx.x, tid = threadIdx.x;
    const int tok0 = p.seq_start[b], n = p.seq_start[b + 1] - tok0;
    llb_grid_dependency_sync();
    if (c * CHUNK >= n) return;
    const int nc = min(CHUNK, n - c * CHUNK), row0 = tok0 + c * CHUNK;
    const int dk = p.dk, dv = p.dv, kh = h / (p.H / p.G), C = 2 * p.G * dk + p.H * dv;
    float* sk = sm;                                        // [16][LD] keys, then keys times the decays since the chunk's start
    float* sq = sk + CHUNK * LD;                           // [16][LD]
    float* sg = sq + CHUNK * LD;                           // [16][LD]
    float* sA = sg + CHUNK * LD;                           // [16][16]
    float* sB = sA + 256;                                  // [16][16]
    float* sT = sB + 256;                                  // [16][16]
    float* sbeta = sT + 256;                               // [16]
    float* rec = p.rec + ((size_t)(chunk_base(tok0, b) + c) * p.H + h) * rec_floats(NP, p.cb);

    if (((dk | C) & 3) == 0) {                             // 16-byte pieces (the operands are this module's own, aligned)
        for (int idx = tid; idx < CHUNK * (DKP / 4); idx += CHUNK_THREADS) {
            const int t = idx / (DKP / 4), i = (idx - t * (DKP / 4)) * 4;
            const bool in = t < nc && i < dk;
            const size_t row = (size_t)(row0 + t);
            const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f), one = make_float4(1.f, 1.f, 1.f, 1.f);
            *reinterpret_cast<float4*>(sq + t * LD + i) = in ? *reinterpret_cast<const float4*>(p.qkv + row * C + kh * dk + i) : zero;
            *reinterpret_cast<float4*>(sk + t * LD + i) = in ? *reinterpret_cast<const float4*>(p.qkv + row * C + (p.G + kh) * dk + i) : zero;
            *reinterpret_cast<float4*>(sg + t * LD + i) = in ? *reinterpret_cast<const float4*>(p.g + (row * p.H + h) * dk + i) : one;
        }
    } else {
        for (int idx = tid; idx < CHUNK * DKP; idx += CHUNK_THREADS) {
            const int t = idx / DKP, i = idx - t * DKP;
            const bool in = t < nc && i < dk;
            const size_t row = (size_t)(row0 + t);
            sq[t * LD + i] = in ? p.qkv[row * C + kh * dk + i] : 0.f;
            sk[t * LD + i] = in ? p.qkv[row * C + (p.G + kh) * dk + i] : 0.f;
            sg[t * LD + i] = in ? p.g[(row * p.H + h) * dk + i] : 1.f;
        }
    }
    if (tid < CHUNK) sbeta[tid] = tid < nc ? p.beta[(size_t)(row0 + tid) * p.H + h] : 0.f;
    __syncthreads();

    // ---- A_ts for s < t and B_ts (q_t in k_t's place) for s <= t: 8 threads share an s, each with every eighth piece of 4
    // channels; their sums are completed by halving (a thread passes on the half it will not keep).  Other places are zero.
    {
        const int s = tid >> 3, part = tid & 7;
        float v[2 * CHUNK];                                // A_ts for t = 0 .. 15, then B_ts
#pragma unroll
        for (int t = 0; t < 2 * CHUNK; ++t) v[t] = 0.f;
        for (int i = part * 4; i < dk; i += 32) {
            float4 run = *reinterpret_cast<const float4*>(sk + s * LD + i);      // k_s times the decays after s, up to t
#pragma unroll
            for (int t = 0; t < CHUNK; ++t) {
                if (t < s) continue;
                if (t > s) {
                    const float4 g = *reinterpret_cast<const float4*>(sg + t * LD + i);
                    const float4 k = *reinterpret_cast<const float4*>(sk + t * LD + i);
                    run.x *= g.x;
                    run.y *= g.y;
                    run.z *= g.z;
                    run.w *= g.w;
                    v[t] = fmaf(k.x, run.x, fmaf(k.y, run.y, fmaf(k.z, run.z, fmaf(k.w, run.w, v[t]))));
                }
                const float4 q = *reinterpret_cast<const float4*>(sq + t * LD + i);
                v[CHUNK + t] = fmaf(q.x, run.x, fmaf(q.y, run.y, fmaf(q.z, run.z, fmaf(q.w, run.w, v[CHUNK + t]))));
            }
        }
#pragma unroll
        for (int half = CHUNK; half >= 4; half >>= 1) {
            const int lane_bit = half / 4;                 // 4, 2, 1
            const bool up = part & lane_bit;
#pragma unroll
            for (int i = 0; i < half; ++i) {
                const float keep = up ? v[i + half] : v[i], send = up ? v[i] : v[i + half];
                v[i] = keep + __shfl_xor_sync(0xffffffffu, send, lane_bit);
            }
        }
        float* dst = (part & 4) ? sB : sA;
        const int t0 = (part & 3) * 4;
#pragma unroll
        for (int i = 0; i < 4; ++i) dst[(t0 + i) * 16 + s] = v[i];
    }
    __syncthreads();
    // ---- T, a column per lane of the first warp; meanwhile the other warps form the products with the running decays
    if (tid < 32) {
        if (tid < CHUNK) {
            float col[CHUNK];
#pragma unroll
            for (int t = 0; t < CHUNK; ++t) {
                float x0 = t == tid ? 1.f : 0.f, x1 = 0.f;
#pragma unroll
                for (int s = 0; s < t; ++s) {
                    if (s & 1) x1 = fmaf(-sA[t * 16 + s], col[s], x1);
                    else x0 = fmaf(-sA[t * 16 + s], col[s], x0);
                }
                col[t] = sbeta[t] * (x0 + x1);
                sT[t * 16 + tid] = col[t];
            }
        }
    } else {
        for (int i = tid - 32; i < DKP; i += CHUNK_THREADS - 32) {
            // the keys as the chunk's end sees them: k_s times the decays after s
            float kv[CHUNK];
            float tail = 1.f;
#pragma unroll
            for (int s = CHUNK - 1; s >= 0; --s) {
                kv[s] = sk[s * LD + i] * tail;
                tail *= sg[s * LD + i];
            }
            const int blk = i >> 4, r = i & 15, half = (r >> 1) & 1, col = (r >> 2) * 2 + (r & 1);
            float4* kf = reinterpret_cast<float4*>(rec + rec_k(NP)) + (blk * 2 + half) * 32 + col * 4;       // lane col * 4 + s / 4
#pragma unroll
            for (int s = 0; s < CHUNK; s += 4) kf[s / 4] = make_float4(kv[s], kv[s + 1], kv[s + 2], kv[s + 3]);
            rec[rec_gam(NP) + i] = tail;
            float head = 1.f;
#pragma unroll
            for (int t = 0; t < CHUNK; ++t) {
                head *= sg[t * LD + i];
                sk[t * LD + i] *= head;
                sq[t * LD + i] *= head;
            }
        }
    }
    __syncthreads();
    // ---- B T, two elements a thread, over A
#pragma unroll
    for (int it = 0; it < 2; ++it) {
        const int t = (tid >> 4) + it * 8, j = tid & 15;
        float x = 0.f;
#pragma unroll
        for (int s = 0; s < CHUNK; ++s) x = fmaf(sB[t * 16 + s], sT[s * 16 + j], x);
        sA[t * 16 + j] = x;
    }
    __syncthreads();
    // ---- W = T (K . G) and the read-out's rows Q . G - B T (K . G), a thread per piece of 4 channels and tile of tokens
#pragma unroll
    for (int it = 0; it < NP / 2; ++it) {
        const int idx = tid + it * CHUNK_THREADS, lane = idx & 31, tile = (idx >> 5) & 1, blk = idx >> 6;
        const int t = frag_index(lane >> 2, tile), i = blk * 16 + (lane & 3) * 4;
        float4 w = make_float4(0.f, 0.f, 0.f, 0.f), x = *reinterpret_cast<const float4*>(sq + t * LD + i);
#pragma unroll
        for (int s = 0; s < CHUNK; s += 4) {
            const float4 f4 = *reinterpret_cast<const float4*>(sT + t * 16 + s), m4 = *reinterpret_cast<const float4*>(sA + t * 16 + s);
            const float f[4] = {f4.x, f4.y, f4.z, f4.w}, m[4] = {m4.x, m4.y, m4.z, m4.w};
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float4 k = *reinterpret_cast<const float4*>(sk + (s + e) * LD + i);
                w.x = fmaf(f[e], k.x, w.x);
                w.y = fmaf(f[e], k.y, w.y);
                w.z = fmaf(f[e], k.z, w.z);
                w.w = fmaf(f[e], k.w, w.w);
                x.x = fmaf(-m[e], k.x, x.x);
                x.y = fmaf(-m[e], k.y, x.y);
                x.z = fmaf(-m[e], k.z, x.z);
                x.w = fmaf(-m[e], k.w, x.w);
            }
        }
        *reinterpret_cast<float4*>(rec + idx * 4) = w;
        *reinterpret_cast<float4*>(rec + rec_q(NP) + idx * 4) = x;
    }
    // ---- T V and B T V, a thread per value column
    for (int col = tid; col < 16 * p.cb; col += CHUNK_THREADS) {
        float v[CHUNK];
#pragma unroll
        for (int t = 0; t < CHUNK; ++t) v[t] = (t < nc && col < dv) ? p.qkv[(size_t)(row0 + t) * C + 2 * p.G * dk + h * dv + col] : 0.f;
        float* block = rec + rec_u(NP) + (col >> 4) * 512;
        const int half = (col >> 3) & 1, lane0 = (col & 7) * 4;
#pragma unroll 1
        for (int t0 = 0; t0 < CHUNK; t0 += 4) {            // (not unrolled: T would be held in registers)
            float u[4], o[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                u[e] = o[e] = 0.f;
#pragma unroll
                for (int s = 0; s < CHUNK; s += 4) {
                    const float4 f = *reinterpret_cast<const float4*>(sT + (t0 + e) * 16 + s);
                    const float4 m = *reinterpret_cast<const float4*>(sA + (t0 + e) * 16 + s);
                    u[e] = fmaf(f.x, v[s], fmaf(f.y, v[s + 1], fmaf(f.z, v[s + 2], fmaf(f.w, v[s + 3], u[e]))));
                    o[e] = fmaf(m.x, v[s], fmaf(m.y, v[s + 1], fmaf(m.z, v[s + 2], fmaf(m.w, v[s + 3], o[e]))));
                }
            }
            *reinterpret_cast<float4*>(block + (half * 32 + lane0) * 4 + t0) = make_float4(u[0], u[1], u[2], u[3]);
            // as the accumulators of two tiles of tokens lie: [tile][lane][row of the pair, token of the pair]
            float* of = block + 256 + (lane0 + t0 / 4) * 4 + half * 2;
            *reinterpret_cast<float2*>(of) = make_float2(o[0], o[1]);
            *reinterpret_cast<float2*>(of + 128) = make_float2(o[2], o[3]);
        }
    }
}

__device__ __forceinline__ void mma_tf32(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// x = hi + lo with hi a TF32 number (its lower 13 bits zero); lo is exact and enters a product with its leading bits.
__device__ __forceinline__ void split(float x, uint32_t& hi, uint32_t& lo) {
    hi = __float_as_uint(x) & 0xffffe000u;
    lo = __float_as_uint(x - __uint_as_float(hi));
}
// An accumulator tile as an A operand: column 2 a of the tile takes the operand's place a, column 2 a + 1 the place a + 4.
__device__ __forceinline__ void split_tile(const float (&c)[4], uint32_t (&hi)[4], uint32_t (&lo)[4]) {
    split(c[0], hi[0], lo[0]);
    split(c[2], hi[1], lo[1]);
    split(c[1], hi[2], lo[2]);
    split(c[3], hi[3], lo[3]);
}
__device__ __forceinline__ void mma_split(float (&c)[4], float (&corr)[4], const uint32_t (&ahi)[4], const uint32_t (&alo)[4], float b0,
                                          float b1) {
    uint32_t h0, l0, h1, l1;
    split(b0, h0, l0);
    split(b1, h1, l1);
    mma_tf32(c, ahi, h0, h1);
    mma_tf32(corr, ahi, l0, l1);
    mma_tf32(corr, alo, h0, h1);
}

constexpr int WALK_K = 4;               // warps that share a head's key channels
constexpr int walk_stages(int npk) { return npk <= 2 ? 4 : 3; }       // records in shared memory
constexpr uint32_t WAIT_LIMIT = 1u << 22;
enum { ERR_DELTA_WAIT = 161 };

__device__ __forceinline__ bool stage_wait(uint32_t bar, uint32_t parity) {
    for (uint32_t i = 0; i < WAIT_LIMIT; ++i) {
        uint32_t done;
        asm volatile("{\n\t.reg .pred p;\n\tmbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\tselp.u32 %0, 1, 0, p;\n\t}"
                     : "=r"(done) : "r"(bar), "r"(parity) : "memory");
        if (done) return true;
    }
    return false;
}

// A block walks the chunks of one head of one sequence with CG x 16 value columns.  Four warps share 16 columns, each with NPK
// blocks of 16 key channels of S; their partial W S_0 and Q S_0 meet in shared memory once a chunk, at the chunk's one barrier.
// A chunk's record arrives by two bulk copies, two or three chunks ahead.
template <int NPK, int CG>
__global__ void __launch_bounds__(CG * WALK_K * 32) delta_walk_kernel(DeltaChunkParams p) {
    extern __shared__ __align__(16) float sm[];
    constexpr int NP = WALK_K * NPK, WALK_STAGES = walk_stages(NPK);
    constexpr int SHARED = rec_u(NP);                      // floats all warps read
    constexpr int STAGE = SHARED + 512 * CG;
    constexpr int EXCH = CG * WALK_K * 128;                // 16-byte pieces of one exchange: [CG][WALK_K][4][32], partial r, o of a warp
    float4* exch = reinterpret_cast<float4*>(sm + WALK_STAGES * STAGE);           // two of them, by turns
    __shared__ __align__(8) unsigned long long bars[WALK_STAGES];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, a4 = lane & 3;
    const int kw = warp % WALK_K, cg = warp / WALK_K;
    const int h = blockIdx.y, b = blockIdx.z, cb0 = blockIdx.x * CG, col0 = (cb0 + cg) * 16;
    const int tok0 = p.seq_start[b], n = p.seq_start[b + 1] - tok0, n_chunks = (n + CHUNK - 1) / CHUNK;
    const uint32_t bar0 = (uint32_t)__cvta_generic_to_shared(bars);
    if (tid == 0) {
        for (int i = 0; i < WALK_STAGES; ++i) asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"(bar0 + i * 8));
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    llb_grid_dependency_sync();
    if (n_chunks == 0) return;
    const int dk = p.dk, dv = p.dv, rf = rec_floats(NP, p.cb), my_cb = min(CG, p.cb - cb0);
    const float* rec = p.rec + ((size_t)chunk_base(tok0, b) * p.H + h) * rf;
    const size_t rec_step = (size_t)p.H * rf;
    const uint32_t sm_addr = (uint32_t)__cvta_generic_to_shared(sm);
    auto fetch = [&](int c) {                              // one thread
        if (c >= n_chunks) return;
        const float* src = rec + (size_t)c * rec_step;
        const uint32_t dst = sm_addr + (uint32_t)((c % WALK_STAGES) * STAGE * 4), bar = bar0 + (c % WALK_STAGES) * 8;
        asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"((uint32_t)(SHARED + my_cb * 512) * 4) : "memory");
        asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                     ::"r"(dst), "l"(src), "r"((uint32_t)SHARED * 4), "r"(bar) : "memory");
        asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                     ::"r"(dst + SHARED * 4), "l"(src + SHARED + cb0 * 512), "r"((uint32_t)(my_cb * 2048)), "r"(bar) : "memory");
    };
    if (tid == 0)
        for (int c = 0; c < WALK_STAGES - 1; ++c) fetch(c);

    // S^T tiles: tile (q, half) holds rows v = g8, g8 + 8 of the columns and channels 16 (kw NPK + q) + 4 a4 + 2 half + {0, 1}
    float S[2 * NPK][4];
    float* st = p.state + ((size_t)p.seq_slot[b] * p.H + h) * dk * dv;
#pragma unroll
    for (int j = 0; j < 2 * NPK; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = (kw * NPK + (j >> 1)) * 16 + 4 * a4 + 2 * (j & 1) + (e & 1), v = col0 + g8 + (e >> 1) * 8;
            S[j][e] = (i < dk && v < dv) ? st[(size_t)i * dv + v] : 0.f;
        }

    // this lane's two results of a chunk, places 2 (32 kw + lane) and + 1 of the accumulators of two tiles: column ocol, tokens ot, ot + 1
    const int place = kw * 32 + lane, ol = (place & 63) >> 1;
    const int ot = 4 * (ol & 3) + 2 * (place >> 6), ocol = col0 + (ol >> 2) + 8 * (place & 1);
    float* out = p.out + (size_t)(tok0 + ot) * p.H * dv + h * dv + ocol;
    const size_t out_row = (size_t)p.H * dv;
    const bool in_col = ocol < dv;
    bool ok = true;
    for (int c = 0; c < n_chunks; ++c, out += CHUNK * out_row) {
        ok = ok && stage_wait(bar0 + (c % WALK_STAGES) * 8, (uint32_t)(c / WALK_STAGES) & 1);
        const float* s = sm + (c % WALK_STAGES) * STAGE;
        const float4* wf = reinterpret_cast<const float4*>(s) + kw * NPK * 64 + lane;
        const float4* qf = reinterpret_cast<const float4*>(s + rec_q(NP)) + kw * NPK * 64 + lane;
        const float4* kf = reinterpret_cast<const float4*>(s + rec_k(NP)) + kw * NPK * 64 + lane;
        // ---- this warp's part of W S_0 and Q S_0 (transposed): [16 columns, 16 tokens] each
        float r[2][4], rc[2][4], o[2][4], oc[2][4];
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
            for (int e = 0; e < 4; ++e) r[t][e] = rc[t][e] = o[t][e] = oc[t][e] = 0.f;
#pragma unroll
        for (int q = 0; q < NPK; ++q) {
            uint32_t h0[4], l0[4], h1[4], l1[4];
            split_tile(S[2 * q], h0, l0);
            split_tile(S[2 * q + 1], h1, l1);
            const float4 w0 = wf[q * 64], w1 = wf[q * 64 + 32], x0 = qf[q * 64], x1 = qf[q * 64 + 32];
            mma_split(r[0], rc[0], h0, l0, w0.x, w0.y);
            mma_split(r[1], rc[1], h0, l0, w1.x, w1.y);
            mma_split(o[0], oc[0], h0, l0, x0.x, x0.y);
            mma_split(o[1], oc[1], h0, l0, x1.x, x1.y);
            mma_split(r[0], rc[0], h1, l1, w0.z, w0.w);
            mma_split(r[1], rc[1], h1, l1, w1.z, w1.w);
            mma_split(o[0], oc[0], h1, l1, x0.z, x0.w);
            mma_split(o[1], oc[1], h1, l1, x1.z, x1.w);
        }
        float4* ex = exch + (c & 1) * EXCH + cg * (WALK_K * 128) + lane;
        ex[kw * 128] = make_float4(r[0][0] + rc[0][0], r[0][1] + rc[0][1], r[0][2] + rc[0][2], r[0][3] + rc[0][3]);
        ex[kw * 128 + 32] = make_float4(r[1][0] + rc[1][0], r[1][1] + rc[1][1], r[1][2] + rc[1][2], r[1][3] + rc[1][3]);
        ex[kw * 128 + 64] = make_float4(o[0][0] + oc[0][0], o[0][1] + oc[0][1], o[0][2] + oc[0][2], o[0][3] + oc[0][3]);
        ex[kw * 128 + 96] = make_float4(o[1][0] + oc[1][0], o[1][1] + oc[1][1], o[1][2] + oc[1][2], o[1][3] + oc[1][3]);
        // what does not wait for the other warps: the decays of the chunk on this warp's part of S
        const float4* gam = reinterpret_cast<const float4*>(s + rec_gam(NP)) + kw * NPK * 4 + a4;
#pragma unroll
        for (int q = 0; q < NPK; ++q) {
            const float4 gm = gam[q * 4];
            S[2 * q][0] *= gm.x;
            S[2 * q][1] *= gm.y;
            S[2 * q][2] *= gm.x;
            S[2 * q][3] *= gm.y;
            S[2 * q + 1][0] *= gm.z;
            S[2 * q + 1][1] *= gm.w;
            S[2 * q + 1][2] *= gm.z;
            S[2 * q + 1][3] *= gm.w;
        }
        float4 ua = make_float4(0.f, 0.f, 0.f, 0.f), ub = ua;
        if (cg < my_cb) {
            const float4* uf = reinterpret_cast<const float4*>(s + SHARED + cg * 512) + lane;
            ua = uf[0];
            ub = uf[32];
        }
        // behind this barrier every warp is done with the chunk before this one, whose stage takes the next record
        // (a thread whose wait ran out waits no more and fetches no more; the walk ends as it would and its result is dropped)
        __syncthreads();
        if (tid == 0 && ok) fetch(c + WALK_STAGES - 1);
        // ---- u = T V - W S_0
        float u0[4], u1[4];
        {
            float4 x = ex[0], y = ex[32];
#pragma unroll
            for (int k = 1; k < WALK_K; ++k) {
                const float4 a = ex[k * 128], d = ex[k * 128 + 32];
                x.x += a.x; x.y += a.y; x.z += a.z; x.w += a.w;
                y.x += d.x; y.y += d.y; y.z += d.z; y.w += d.w;
            }
            u0[0] = ua.x - x.x; u0[1] = ua.y - x.y; u0[2] = ub.x - x.z; u0[3] = ub.y - x.w;
            u1[0] = ua.z - y.x; u1[1] = ua.w - y.y; u1[2] = ub.z - y.z; u1[3] = ub.w - y.w;
        }
        uint32_t uh[2][4], ul[2][4];
        split_tile(u0, uh[0], ul[0]);
        split_tile(u1, uh[1], ul[1]);
        // ---- S <- diag(G) S + K^T u
#pragma unroll
        for (int q = 0; q < NPK; ++q) {
            float corr[2][4];
#pragma unroll
            for (int half = 0; half < 2; ++half)
#pragma unroll
                for (int e = 0; e < 4; ++e) corr[half][e] = 0.f;
            const float4 k0 = kf[q * 64], k1 = kf[q * 64 + 32];
            mma_split(S[2 * q], corr[0], uh[0], ul[0], k0.x, k0.y);
            mma_split(S[2 * q + 1], corr[1], uh[0], ul[0], k1.x, k1.y);
            mma_split(S[2 * q], corr[0], uh[1], ul[1], k0.z, k0.w);
            mma_split(S[2 * q + 1], corr[1], uh[1], ul[1], k1.z, k1.w);
#pragma unroll
            for (int half = 0; half < 2; ++half)
#pragma unroll
                for (int e = 0; e < 4; ++e) S[2 * q + half][e] += corr[half][e];
        }
        // ---- o = (Q . G - B W) S_0 + B T V, a quarter of the places for each of the four warps
        if (in_col) {
            const float2* e2 = reinterpret_cast<const float2*>(ex - lane) + 128 + place;
            float2 x = reinterpret_cast<const float2*>(s + SHARED + cg * 512 + 256)[place];
#pragma unroll
            for (int k = 0; k < WALK_K; ++k) {
                const float2 a = e2[k * 256];
                x.x += a.x;
                x.y += a.y;
            }
            const int tl = c * CHUNK + ot;
            if (tl < n) out[0] = x.x;
            if (tl + 1 < n) out[out_row] = x.y;
        }
    }
    if (__syncthreads_or(!ok)) {                           // a bounded wait ran out: the copies in flight get a bounded time to land
        if (tid == 0) {
            atomicExch(p.err, ERR_DELTA_WAIT);
            for (int i = 0; i < 1000; ++i) __nanosleep(1000);
        }
        return;
    }
#pragma unroll
    for (int j = 0; j < 2 * NPK; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = (kw * NPK + (j >> 1)) * 16 + 4 * a4 + 2 * (j & 1) + (e & 1), v = col0 + g8 + (e >> 1) * 8;
            if (i < dk && v < dv) st[(size_t)i * dv + v] = S[j][e];
        }
}

int set_smem(const void* kernel, bool& configured, size_t smem) {
    if (configured) return 0;
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    configured = true;                                     // once per kernel: not repeated inside a graph capture
    return 0;
}

template <int KS, int KPT>
int launch_scan(const DeltaScanParams& p, int B, cudaStream_t stream) {
    auto k = delta_scan_kernel<KS, KPT>;
    constexpr int COLS = SCAN_THREADS / KS;
    constexpr size_t smem = (size_t)(3 * SCAN_STAGE * KS * (KPT + scan_pad(KPT)) + SCAN_STAGE * COLS + SCAN_STAGE) * sizeof(float);
    static bool configured = false;
    if (int rc = set_smem((const void*)k, configured, smem)) return rc;
    llb_launch(k, dim3((p.dv + COLS - 1) / COLS, p.H, B), dim3(SCAN_THREADS), smem, stream, p);
    return llb_status();
}
template <int KS>
int launch_scan_ks(const DeltaScanParams& p, int B, cudaStream_t stream) {
    const int kpt = (p.dk + KS - 1) / KS;
    if (kpt <= 4) return launch_scan<KS, 4>(p, B, stream);
    if (kpt <= 8) return launch_scan<KS, 8>(p, B, stream);
    if (kpt <= 16) return launch_scan<KS, 16>(p, B, stream);
    if constexpr (KS <= 8) {
        if (kpt <= 32) return launch_scan<KS, 32>(p, B, stream);
    }
    if constexpr (KS <= 4) {
        if (kpt <= 64) return launch_scan<KS, 64>(p, B, stream);
    }
    return (int)cudaErrorInvalidValue;
}

template <int NPK, int CG>
int launch_walk(const DeltaChunkParams& p, int B, cudaStream_t stream) {
    auto k = delta_walk_kernel<NPK, CG>;
    constexpr size_t smem = (size_t)(walk_stages(NPK) * (rec_u(WALK_K * NPK) + 512 * CG) + 2 * CG * WALK_K * 512) * sizeof(float);
    static_assert(smem <= 227 * 1024, "the stages fit an SM");
    static bool configured = false;
    if (int rc = set_smem((const void*)k, configured, smem)) return rc;
    llb_launch(k, dim3((p.cb + CG - 1) / CG, p.H, B), dim3(CG * WALK_K * 32), smem, stream, p);
    return llb_status();
}

template <int NPK>
int launch_chunked(const DeltaChunkParams& p, int B, int max_new, int sms, cudaStream_t stream) {
    auto k = delta_chunk_kernel<NPK>;
    constexpr size_t smem = (size_t)(3 * CHUNK * (64 * NPK + 4) + 768 + CHUNK) * sizeof(float);
    static bool configured = false;
    if (int rc = set_smem((const void*)k, configured, smem)) return rc;
    llb_launch(k, dim3((max_new + CHUNK - 1) / CHUNK, p.H, B), dim3(CHUNK_THREADS), smem, stream, p);
    if (int rc = llb_status()) return rc;
    // two groups of columns a block read a chunk's fragments once for both, where there are blocks enough without
    if ((long long)((p.cb + 1) / 2) * p.H * B * 4 >= 3ll * sms) return launch_walk<NPK, 2>(p, B, stream);
    return launch_walk<NPK, 1>(p, B, stream);
}

int channel_blocks(int dk) { return (dk + 63) / 64; }      // NPK

bool sizes_ok(int G, int H, int dk, int dv, int B) {
    return G > 0 && H > 0 && H % G == 0 && dk > 0 && dk <= 256 && dv > 0 && H <= 65535 && B <= 65535;
}

}  // namespace

LLB_API int llb_delta_prep(DeltaPrepParams p, int B, int max_new, cudaStream_t stream) {
    if (B == 0 || max_new == 0) return 0;
    if (!sizes_ok(p.G, p.H, p.dk, p.dv, B) || p.dv > 256 || p.taps < 1 || 2 * p.G + 2 * p.H > 65535) return (int)cudaErrorInvalidValue;
    const int run = PREP_WARPS * prep_run(p.taps), C = 2 * p.G * p.dk + p.H * p.dv;
    p.vec = p.ld % 4 == 0 && C % 4 == 0 && p.dk % 4 == 0 && p.dv % 4 == 0 &&
            !(((uintptr_t)p.proj | (uintptr_t)p.conv_w | (uintptr_t)p.conv_state | (uintptr_t)p.out) & 15);
    const dim3 grid((max_new + run - 1) / run, 2 * p.G + 2 * p.H, B), block(PREP_WARPS * 32);
    if (p.taps == 4 && p.fast) llb_launch(delta_prep_kernel<4, true>, grid, block, 0, stream, p);
    else if (p.taps == 4) llb_launch(delta_prep_kernel<4, false>, grid, block, 0, stream, p);
    else if (p.fast) llb_launch(delta_prep_kernel<0, true>, grid, block, 0, stream, p);
    else llb_launch(delta_prep_kernel<0, false>, grid, block, 0, stream, p);
    return llb_status();
}

// The recurrence over the new tokens of every sequence of the step.  More lanes share a column (fewer columns a block, more
// blocks) while the blocks would not fill the device and a lane still keeps eight channels.
LLB_API int llb_delta_scan(DeltaScanParams p, int B, int sms, cudaStream_t stream) {
    if (B == 0) return 0;
    if (!sizes_ok(p.G, p.H, p.dk, p.dv, B)) return (int)cudaErrorInvalidValue;
    int ks = 4;
    while (ks < 16 && (long long)((p.dv + 128 / ks - 1) / (128 / ks)) * p.H * B < sms && p.dk >= 8 * ks) ks *= 2;
    if (ks == 4) return launch_scan_ks<4>(p, B, stream);
    if (ks == 8) return launch_scan_ks<8>(p, B, stream);
    return launch_scan_ks<16>(p, B, stream);
}

// Floats of the scratch that llb_delta_chunked needs for T packed tokens of B sequences.
LLB_API long long llb_delta_scratch(int T, int B, int H, int dk, int dv) {
    return (long long)(T / CHUNK + B + 1) * H * rec_floats(4 * channel_blocks(dk), (dv + 15) / 16);
}

// The same recurrence in chunks; p.rec holds llb_delta_scratch() floats, p.cb is set here.
LLB_API int llb_delta_chunked(DeltaChunkParams p, int B, int max_new, int sms, cudaStream_t stream) {
    if (B == 0 || max_new == 0) return 0;
    if (!sizes_ok(p.G, p.H, p.dk, p.dv, B) || (((uintptr_t)p.rec | (uintptr_t)p.qkv | (uintptr_t)p.g) & 15)) return (int)cudaErrorInvalidValue;
    p.cb = (p.dv + 15) / 16;
    switch (channel_blocks(p.dk)) {
        case 1: return launch_chunked<1>(p, B, max_new, sms, stream);
        case 2: return launch_chunked<2>(p, B, max_new, sms, stream);
        case 3: return launch_chunked<3>(p, B, max_new, sms, stream);
        case 4: return launch_chunked<4>(p, B, max_new, sms, stream);
    }
    return (int)cudaErrorInvalidValue;
}
