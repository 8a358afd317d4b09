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
//                      so all that does not contain S_0 (A, T, W = T (K . G), T V, the readout's own matrix) is computed for
//                      every chunk side by side (delta_chunk), and only three matrix products with the state a chunk remain
//                      sequential (delta_walk).  Decays are only ever multiplied up, never divided, so a channel that
//                      forgets at once costs nothing but its products.
//                      delta_walk runs on the tensor cores: a warp owns 16 value columns of S as accumulator fragments, which
//                      are the A operand of the next chunk's products without leaving the registers.  Every float32 operand
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
    const int* tok_seq;       // [T]
    const int* seq_start;     // [B + 1]
    const int* seq_slot;      // [B]
    float* out;               // [T, C]
    float* beta;              // [T, H]
    int T, G, H, dk, dv, taps;
    float q_scale;
    int single;               // every sequence brings one token: the warp that read a channel's inputs shifts them itself
};

__device__ __forceinline__ float silu(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

constexpr int PREP_WARPS = 4;
constexpr int MAX_PER = 8;              // channels of a head a lane holds: heads of up to 256

__global__ void __launch_bounds__(PREP_WARPS * 32) delta_prep_kernel(DeltaPrepParams p) {
    const int lane = threadIdx.x & 31;
    const int t = blockIdx.x * PREP_WARPS + (threadIdx.x >> 5), unit = blockIdx.y;
    const int C = 2 * p.G * p.dk + p.H * p.dv;
    llb_grid_dependency_sync();
    if (t >= p.T) return;
    if (unit >= 2 * p.G + p.H) {                           // a head's decays and its step size
        const int h = unit - 2 * p.G - p.H;
        const float rate = expf(p.a_log[h]);
        float* z = p.z + ((size_t)t * p.H + h) * p.dk;
        for (int i = lane; i < p.dk; i += 32) z[i] = expf(-rate * softplus(z[i]));
        if (lane == 0) p.beta[(size_t)t * p.H + h] = 1.0f / (1.0f + expf(-p.proj[(size_t)t * p.ld + C + h]));
        return;
    }
    const bool is_qk = unit < 2 * p.G;
    const int d = is_qk ? p.dk : p.dv;
    const int c0 = is_qk ? unit * p.dk : 2 * p.G * p.dk + (unit - 2 * p.G) * p.dv;
    const int b = p.tok_seq[t], at = t - p.seq_start[b], back = p.taps - 1;
    float* st = p.conv_state + (size_t)p.seq_slot[b] * back * C + c0;
    const float* x = p.proj + (size_t)t * p.ld + c0;
    float v[MAX_PER];
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < MAX_PER; ++e) {
        const int i = lane + e * 32;
        v[e] = 0.f;
        if (i < d) {
            float acc = 0.f;
#pragma unroll 4
            for (int j = 0; j < p.taps; ++j) {
                const int r = at - back + j;               // the input's place among the step's tokens of the sequence
                const float in = r >= 0 ? x[(ptrdiff_t)(j - back) * p.ld + i] : st[(size_t)(r + back) * C + i];
                acc = fmaf(p.conv_w[(size_t)j * C + c0 + i], in, acc);
            }
            v[e] = silu(acc);
            ss = fmaf(v[e], v[e], ss);
            if (p.single) {
                for (int j = 0; j + 1 < back; ++j) st[(size_t)j * C + i] = st[(size_t)(j + 1) * C + i];
                if (back > 0) st[(size_t)(back - 1) * C + i] = x[i];
            }
        }
    }
    float f = 1.f;
    if (is_qk) {
        f = 1.0f / sqrtf(warp_sum(ss) + UNIT_EPS);
        if (unit < p.G) f *= p.q_scale;
    }
    float* out = p.out + (size_t)t * C + c0;
#pragma unroll
    for (int e = 0; e < MAX_PER; ++e)
        if (lane + e * 32 < d) out[lane + e * 32] = v[e] * f;
}

// The inputs that the next step's convolution needs: the last taps - 1 of (old state, the step's tokens).  A thread per
// sequence and channel; ascending, so that what is still needed of the old state has not been overwritten.
__global__ void __launch_bounds__(256) delta_conv_state_kernel(DeltaPrepParams p) {
    const int C = 2 * p.G * p.dk + p.H * p.dv, back = p.taps - 1;
    const int c = blockIdx.x * blockDim.x + threadIdx.x, b = blockIdx.y;
    llb_grid_dependency_sync();
    if (c >= C) return;
    const int tok0 = p.seq_start[b], n = p.seq_start[b + 1] - tok0;
    float* st = p.conv_state + (size_t)p.seq_slot[b] * back * C + c;
    for (int j = 0; j < back; ++j) {
        const int r = n - back + j;
        st[(size_t)j * C] = r >= 0 ? p.proj[(size_t)(tok0 + r) * p.ld + c] : st[(size_t)(j + n) * C];
    }
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
    int G, H, dk, dv;
    int np, cb;               // blocks of 16 key channels (padded), blocks of 16 value columns
};

// What delta_chunk leaves for one chunk of one head, in floats.  W, Q and K are stored as the fragments that delta_walk
// multiplies with: 16-byte pieces, lane by lane.
__host__ __device__ constexpr int rec_w(int) { return 0; }
__host__ __device__ constexpr int rec_q(int np) { return 256 * np; }
__host__ __device__ constexpr int rec_k(int np) { return 512 * np; }
__host__ __device__ constexpr int rec_gam(int np) { return 768 * np; }
__host__ __device__ constexpr int rec_b(int np) { return 784 * np; }
__host__ __device__ constexpr int rec_u(int np) { return 784 * np + 256; }
__host__ __device__ constexpr int rec_floats(int np, int cb) { return rec_u(np) + 256 * cb; }

// The first chunk's place among all chunks of the step: sequences need not start at multiples of 16, and two never collide.
__device__ __forceinline__ int chunk_base(int tok0, int b) { return tok0 / CHUNK + b; }

// Fragment order.  A tile of 8 columns of the chunk's tokens holds the tokens 4 (n / 2) + n % 2 + 2 tile, n = 0 .. 7, and a
// tile of 8 key channels of block p the channels 16 p + 4 (n / 2) + n % 2 + 2 half: so the two TF32 steps of a pair of tiles
// find their operands in one 16-byte piece.
__device__ __forceinline__ int frag_index(int n, int tile) { return 4 * (n >> 1) + (n & 1) + 2 * tile; }

__global__ void __launch_bounds__(CHUNK_THREADS) delta_chunk_kernel(DeltaChunkParams p) {
    extern __shared__ __align__(16) float sm[];
    const int b = blockIdx.z, h = blockIdx.y, c = blockIdx.x, tid = threadIdx.x;
    llb_grid_dependency_sync();
    const int tok0 = p.seq_start[b], n = p.seq_start[b + 1] - tok0;
    if (c * CHUNK >= n) return;
    const int nc = min(CHUNK, n - c * CHUNK), row0 = tok0 + c * CHUNK;
    const int dk = p.dk, dv = p.dv, kh = h / (p.H / p.G), C = 2 * p.G * dk + p.H * dv;
    const int DKP = 16 * p.np, LD = DKP + 4;               // rows 16-byte aligned; a step of 4 banks from row to row
    float* sk = sm;                                        // [16][LD] keys, then keys times the decays since the chunk's start
    float* sq = sk + CHUNK * LD;                           // [16][LD]
    float* sg = sq + CHUNK * LD;                           // [16][LD]
    float* sA = sg + CHUNK * LD;                           // [16][16]
    float* sB = sA + 256;                                  // [16][16]
    float* sT = sB + 256;                                  // [16][16]
    float* sbeta = sT + 256;                               // [16]
    float* rec = p.rec + ((size_t)(chunk_base(tok0, b) + c) * p.H + h) * rec_floats(p.np, p.cb);

    for (int idx = tid; idx < CHUNK * DKP; idx += CHUNK_THREADS) {
        const int t = idx / DKP, i = idx - t * DKP;
        const bool in = t < nc && i < dk;
        const size_t row = (size_t)(row0 + t);
        sq[t * LD + i] = in ? p.qkv[row * C + kh * dk + i] : 0.f;
        sk[t * LD + i] = in ? p.qkv[row * C + (p.G + kh) * dk + i] : 0.f;
        sg[t * LD + i] = in ? p.g[(row * p.H + h) * dk + i] : 1.f;
    }
    if (tid < CHUNK) sbeta[tid] = tid < nc ? p.beta[(size_t)(row0 + tid) * p.H + h] : 0.f;
    for (int idx = tid; idx < 512; idx += CHUNK_THREADS) sA[idx] = 0.f;          // A and B
    __syncthreads();

    // ---- A_ts and B_ts (with q_t in k_t's place, s <= t): 8 threads share an s, each with every eighth piece of 4 channels
    {
        const int s = tid >> 3, part = tid & 7;
        float a[CHUNK], bq[CHUNK];
#pragma unroll
        for (int t = 0; t < CHUNK; ++t) a[t] = bq[t] = 0.f;
        for (int i = part * 4; i < DKP; i += 32) {
            float4 run = *reinterpret_cast<const float4*>(sk + s * LD + i);      // k_s times the decays after s, up to t
#pragma unroll
            for (int t = 0; t < CHUNK; ++t) {
                if (t < s) continue;
                const float4 q = *reinterpret_cast<const float4*>(sq + t * LD + i);
                if (t > s) {
                    const float4 g = *reinterpret_cast<const float4*>(sg + t * LD + i);
                    const float4 k = *reinterpret_cast<const float4*>(sk + t * LD + i);
                    run.x *= g.x; run.y *= g.y; run.z *= g.z; run.w *= g.w;
                    a[t] = fmaf(k.x, run.x, fmaf(k.y, run.y, fmaf(k.z, run.z, fmaf(k.w, run.w, a[t]))));
                }
                bq[t] = fmaf(q.x, run.x, fmaf(q.y, run.y, fmaf(q.z, run.z, fmaf(q.w, run.w, bq[t]))));
            }
        }
#pragma unroll
        for (int t = 0; t < CHUNK; ++t) {
#pragma unroll
            for (int o = 1; o < 8; o <<= 1) {
                a[t] += __shfl_xor_sync(0xffffffffu, a[t], o);
                bq[t] += __shfl_xor_sync(0xffffffffu, bq[t], o);
            }
            if (part == (t & 7) && t >= s) {
                sA[t * 16 + s] = a[t];
                sB[t * 16 + s] = bq[t];
            }
        }
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
            float kv[CHUNK], gv[CHUNK];
#pragma unroll
            for (int t = 0; t < CHUNK; ++t) {
                kv[t] = sk[t * LD + i];
                gv[t] = sg[t * LD + i];
            }
            // the keys as the chunk's end sees them: k_s times the decays after s
            float tail = 1.f;
            const int blk = i >> 4, r = i & 15, half = (r >> 1) & 1, col = (r >> 2) * 2 + (r & 1);
            float* kf = rec + rec_k(p.np) + ((blk * 2 + half) * 32 + col * 4) * 4;
#pragma unroll
            for (int s = CHUNK - 1; s >= 0; --s) {
                kf[s] = kv[s] * tail;                      // lane col * 4 + s / 4, element s % 4
                tail *= gv[s];
            }
            rec[rec_gam(p.np) + i] = tail;
            float head = 1.f;
#pragma unroll
            for (int t = 0; t < CHUNK; ++t) {
                head *= gv[t];
                sk[t * LD + i] = kv[t] * head;
                sq[t * LD + i] *= head;
            }
        }
    }
    __syncthreads();
    // ---- W = T (K . G) and the read-out's rows, a thread per piece of 4 channels and tile of tokens
    for (int idx = tid; idx < p.np * 64; idx += CHUNK_THREADS) {
        const int lane = idx & 31, tile = (idx >> 5) & 1, blk = idx >> 6;
        const int t = frag_index(lane >> 2, tile), i = blk * 16 + (lane & 3) * 4;
        float4 w = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int s = 0; s <= t; ++s) {
            const float f = sT[t * 16 + s];
            const float4 k = *reinterpret_cast<const float4*>(sk + s * LD + i);
            w.x = fmaf(f, k.x, w.x);
            w.y = fmaf(f, k.y, w.y);
            w.z = fmaf(f, k.z, w.z);
            w.w = fmaf(f, k.w, w.w);
        }
        *reinterpret_cast<float4*>(rec + rec_w(p.np) + idx * 4) = w;
        *reinterpret_cast<float4*>(rec + rec_q(p.np) + idx * 4) = *reinterpret_cast<const float4*>(sq + t * LD + i);
    }
    if (tid < 64) {
        const int lane = tid & 31, t = frag_index(lane >> 2, tid >> 5);
        *reinterpret_cast<float4*>(rec + rec_b(p.np) + tid * 4) = *reinterpret_cast<const float4*>(sB + t * 16 + (lane & 3) * 4);
    }
    // ---- T V, a thread per value column
    for (int col = tid; col < 16 * p.cb; col += CHUNK_THREADS) {
        float v[CHUNK];
#pragma unroll
        for (int t = 0; t < CHUNK; ++t) v[t] = (t < nc && col < dv) ? p.qkv[(size_t)(row0 + t) * C + 2 * p.G * dk + h * dv + col] : 0.f;
        float* uf = rec + rec_u(p.np) + (((col >> 4) * 2 + ((col >> 3) & 1)) * 32 + (col & 7) * 4) * 4;
#pragma unroll
        for (int t = 0; t < CHUNK; ++t) {
            float x = 0.f;
#pragma unroll
            for (int s = 0; s <= t; ++s) x = fmaf(sT[t * 16 + s], v[s], x);
            uf[t] = x;
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

constexpr int WALK_WARPS = 4;
constexpr int WALK_STAGES = 3;

// A block walks the chunks of one head of one sequence with 4 x 16 value columns; warp w owns columns [16 w, 16 w + 16).
template <int NP>
__global__ void __launch_bounds__(WALK_WARPS * 32) delta_walk_kernel(DeltaChunkParams p) {
    extern __shared__ __align__(16) float sm[];
    constexpr int SHARED = rec_u(NP);                      // floats all warps read
    constexpr int STAGE = SHARED + 256 * WALK_WARPS;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, a4 = lane & 3;
    const int h = blockIdx.y, b = blockIdx.z, cb0 = blockIdx.x * WALK_WARPS, cbw = cb0 + warp;
    llb_grid_dependency_sync();
    const int tok0 = p.seq_start[b], n = p.seq_start[b + 1] - tok0, n_chunks = (n + CHUNK - 1) / CHUNK;
    if (n_chunks == 0) return;
    const int dk = p.dk, dv = p.dv, rf = rec_floats(NP, p.cb), my_cb = min(WALK_WARPS, p.cb - cb0);
    const float* rec = p.rec + ((size_t)chunk_base(tok0, b) * p.H + h) * rf;
    const size_t rec_step = (size_t)p.H * rf;
    const uint32_t sm_addr = (uint32_t)__cvta_generic_to_shared(sm);
    auto fetch = [&](int c) {
        if (c < n_chunks) {
            const float* src = rec + (size_t)c * rec_step;
            const uint32_t dst = sm_addr + (uint32_t)((c % WALK_STAGES) * STAGE * 4);
            for (int i = tid; i < SHARED / 4; i += WALK_WARPS * 32)
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst + i * 16), "l"(src + i * 4) : "memory");
            for (int i = tid; i < my_cb * 64; i += WALK_WARPS * 32)
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst + (SHARED + i * 4) * 4), "l"(src + SHARED + cb0 * 256 + i * 4) : "memory");
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    for (int c = 0; c < WALK_STAGES - 1; ++c) fetch(c);

    // S^T tiles: tile (p, half) holds rows v = g8, g8 + 8 of the warp's columns and channels 16 p + 4 a4 + 2 half + {0, 1}
    float S[2 * NP][4];
    float* st = p.state + ((size_t)p.seq_slot[b] * p.H + h) * dk * dv;
#pragma unroll
    for (int j = 0; j < 2 * NP; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = (j >> 1) * 16 + 4 * a4 + 2 * (j & 1) + (e & 1), v = cbw * 16 + g8 + (e >> 1) * 8;
            S[j][e] = (i < dk && v < dv) ? st[(size_t)i * dv + v] : 0.f;
        }

    for (int c = 0; c < n_chunks; ++c) {
        asm volatile("cp.async.wait_group %0;" ::"n"(WALK_STAGES - 2) : "memory");
        __syncthreads();                                   // the chunk has landed, and its predecessor's stage is free
        fetch(c + WALK_STAGES - 1);
        const float* s = sm + (c % WALK_STAGES) * STAGE;
        const float4* wf = reinterpret_cast<const float4*>(s + rec_w(NP)) + lane;
        const float4* qf = reinterpret_cast<const float4*>(s + rec_q(NP)) + lane;
        const float4* kf = reinterpret_cast<const float4*>(s + rec_k(NP)) + lane;
        // ---- W S_0 and Q S_0 (transposed): [16 columns, 16 tokens] each
        float r[2][4], rc[2][4], o[2][4], oc[2][4];
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
            for (int e = 0; e < 4; ++e) r[t][e] = rc[t][e] = o[t][e] = oc[t][e] = 0.f;
#pragma unroll
        for (int q = 0; q < NP; ++q) {
            uint32_t h0[4], l0[4], h1[4], l1[4];
            split_tile(S[2 * q], h0, l0);
            split_tile(S[2 * q + 1], h1, l1);
#pragma unroll
            for (int t = 0; t < 2; ++t) {
                const float4 w = wf[(q * 2 + t) * 32], x = qf[(q * 2 + t) * 32];
                mma_split(r[t], rc[t], h0, l0, w.x, w.y);
                mma_split(o[t], oc[t], h0, l0, x.x, x.y);
                mma_split(r[t], rc[t], h1, l1, w.z, w.w);
                mma_split(o[t], oc[t], h1, l1, x.z, x.w);
            }
        }
        // ---- u = T V - W S_0
        if (warp < my_cb) {
            const float4* uf = reinterpret_cast<const float4*>(s + SHARED + warp * 256) + lane;
            const float4 ua = uf[0], ub = uf[32];
            r[0][0] = ua.x - (r[0][0] + rc[0][0]);
            r[0][1] = ua.y - (r[0][1] + rc[0][1]);
            r[1][0] = ua.z - (r[1][0] + rc[1][0]);
            r[1][1] = ua.w - (r[1][1] + rc[1][1]);
            r[0][2] = ub.x - (r[0][2] + rc[0][2]);
            r[0][3] = ub.y - (r[0][3] + rc[0][3]);
            r[1][2] = ub.z - (r[1][2] + rc[1][2]);
            r[1][3] = ub.w - (r[1][3] + rc[1][3]);
        }
        uint32_t uh[2][4], ul[2][4];
        split_tile(r[0], uh[0], ul[0]);
        split_tile(r[1], uh[1], ul[1]);
        // ---- o = Q S_0 + B u
        {
            const float4* bf = reinterpret_cast<const float4*>(s + rec_b(NP)) + lane;
#pragma unroll
            for (int t = 0; t < 2; ++t) {
                const float4 x = bf[t * 32];
                mma_split(o[t], oc[t], uh[0], ul[0], x.x, x.y);
                mma_split(o[t], oc[t], uh[1], ul[1], x.z, x.w);
            }
        }
        // ---- S <- diag(G) S + K^T u
        const float4* gam = reinterpret_cast<const float4*>(s + rec_gam(NP)) + a4;
#pragma unroll
        for (int q = 0; q < NP; ++q) {
            const float4 gm = gam[q * 4];
            float corr[2][4];
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                float (&T)[4] = S[2 * q + half];
                const float ga = half ? gm.z : gm.x, gb = half ? gm.w : gm.y;
                T[0] *= ga;
                T[1] *= gb;
                T[2] *= ga;
                T[3] *= gb;
#pragma unroll
                for (int e = 0; e < 4; ++e) corr[half][e] = 0.f;
                const float4 k = kf[(q * 2 + half) * 32];
                mma_split(T, corr[half], uh[0], ul[0], k.x, k.y);
                mma_split(T, corr[half], uh[1], ul[1], k.z, k.w);
#pragma unroll
                for (int e = 0; e < 4; ++e) T[e] += corr[half][e];
            }
        }
        // ---- the chunk's results: this lane's tokens are 4 a4 + {0, 1} (tile 0) and 4 a4 + {2, 3} (tile 1)
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int tl = c * CHUNK + 4 * a4 + 2 * t + (e & 1), v = cbw * 16 + g8 + (e >> 1) * 8;
                if (tl < n && v < dv) p.out[(size_t)(tok0 + tl) * p.H * dv + h * dv + v] = o[t][e] + oc[t][e];
            }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
    for (int j = 0; j < 2 * NP; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = (j >> 1) * 16 + 4 * a4 + 2 * (j & 1) + (e & 1), v = cbw * 16 + g8 + (e >> 1) * 8;
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

template <int NP>
int launch_walk(const DeltaChunkParams& p, int B, cudaStream_t stream) {
    auto k = delta_walk_kernel<NP>;
    constexpr size_t smem = (size_t)WALK_STAGES * (rec_u(NP) + 256 * WALK_WARPS) * sizeof(float);
    static_assert(smem <= 227 * 1024, "the stages fit an SM");
    static bool configured = false;
    if (int rc = set_smem((const void*)k, configured, smem)) return rc;
    llb_launch(k, dim3((p.cb + WALK_WARPS - 1) / WALK_WARPS, p.H, B), dim3(WALK_WARPS * 32), smem, stream, p);
    return llb_status();
}

// blocks of 16 key channels a kernel is built for
int padded_blocks(int dk) {
    const int np = (dk + 15) / 16;
    for (int v : {1, 2, 3, 4, 6, 8, 12, 16})
        if (np <= v) return v;
    return 0;
}

bool sizes_ok(int G, int H, int dk, int dv, int B) {
    return G > 0 && H > 0 && H % G == 0 && dk > 0 && dk <= 256 && dv > 0 && H <= 65535 && B <= 65535;
}

}  // namespace

LLB_API int llb_delta_prep(DeltaPrepParams p, int B, cudaStream_t stream) {
    if (p.T == 0) return 0;
    if (!sizes_ok(p.G, p.H, p.dk, p.dv, B) || p.dv > 256 || p.taps < 1 || 2 * p.G + 2 * p.H > 65535) return (int)cudaErrorInvalidValue;
    llb_launch(delta_prep_kernel, dim3((p.T + PREP_WARPS - 1) / PREP_WARPS, 2 * p.G + 2 * p.H), dim3(PREP_WARPS * 32), 0, stream, p);
    if (!p.single && p.taps > 1) {
        const int C = 2 * p.G * p.dk + p.H * p.dv;
        llb_launch(delta_conv_state_kernel, dim3((C + 255) / 256, B), dim3(256), 0, stream, p);
    }
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

// Floats of the scratch that llb_delta_chunked needs for T packed tokens of B sequences (0: it does not take these sizes).
LLB_API long long llb_delta_scratch(int T, int B, int H, int dk, int dv) {
    if (dk <= 0 || dk > 256 || dv <= 0) return 0;
    return (long long)(T / CHUNK + B + 1) * H * rec_floats(padded_blocks(dk), (dv + 15) / 16);
}

// The same recurrence in chunks; p.rec holds llb_delta_scratch() floats, p.np and p.cb are set here.
LLB_API int llb_delta_chunked(DeltaChunkParams p, int B, int max_new, cudaStream_t stream) {
    if (B == 0 || max_new == 0) return 0;
    if (!sizes_ok(p.G, p.H, p.dk, p.dv, B) || ((uintptr_t)p.rec & 15)) return (int)cudaErrorInvalidValue;
    p.np = padded_blocks(p.dk);
    p.cb = (p.dv + 15) / 16;
    const size_t smem = (size_t)(3 * CHUNK * (16 * p.np + 4) + 768 + CHUNK) * sizeof(float);
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(delta_chunk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    llb_launch(delta_chunk_kernel, dim3((max_new + CHUNK - 1) / CHUNK, p.H, B), dim3(CHUNK_THREADS), smem, stream, p);
    if (int rc = llb_status()) return rc;
    switch (p.np) {
        case 1: return launch_walk<1>(p, B, stream);
        case 2: return launch_walk<2>(p, B, stream);
        case 3: return launch_walk<3>(p, B, stream);
        case 4: return launch_walk<4>(p, B, stream);
        case 6: return launch_walk<6>(p, B, stream);
        case 8: return launch_walk<8>(p, B, stream);
        case 12: return launch_walk<12>(p, B, stream);
        case 16: return launch_walk<16>(p, B, stream);
    }
    return (int)cudaErrorInvalidValue;
}
