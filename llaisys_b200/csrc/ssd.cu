// Structured state space duality (Dao and Gu, "Transformers are SSMs", 2024): a recurrent mixer whose memory per head is a matrix
// S [N, P] in float32 with one decay per head and token:
//
//     dt_t = softplus(dt'_t + bias_h),  S_t = exp(-exp(A_h) dt_t) S_(t-1) + dt_t B_t x_t^T,  y_t = S_t^T C_t + D_h x_t
//
// x has H heads of P channels, B and C G groups of N (head h reads group h / (H / G)); a row of the operand holds x, B, C.
//
//   ssd_scan        token by token in float32: single tokens, short steps and the 32-bit path
//   ssd_chunk_*     long steps in chunks of 64 tokens on the tensor cores.  With c_t the sum of the log decays from the chunk's
//                   start to token t and S_0 the state at its start
//                       y_t = exp(c_t) S_0^T C_t + sum_(s <= t) exp(c_t - c_s) dt_s (C_t . B_s) x_s + D x_t
//                       S_end = exp(c_end) S_0 + sum_s exp(c_end - c_s) dt_s B_s x_s^T
//                   ssd_chunk_state forms every chunk's own sum, ssd_chunk_prefix walks the chunks of a sequence element by
//                   element (and leaves the states that chunks start with), ssd_chunk_out the results.  x, B and C are
//                   bfloat16 and enter the products exactly; a float32 factor (the state, a weighted score, a weighted x) is
//                   split into two bfloat16 numbers, so that a product keeps about 16 of its bits; sums are float32.
//   gated_group_norm   what follows: y * silu(z), normed in equal parts of the row, times a weight.
#include "common.cuh"

namespace {

struct SsdParams {
    const void* xbc;          // [T, ld]: x (H P), B (G N), C (G N)
    int ld;
    const float* dt;          // [T, dt_ld] logits, H of them a row
    int dt_ld;
    const float* dt_bias;     // [H]
    const float* a_log;       // [H]
    const float* skip;        // [H] (D)
    float* state;             // [slots, H N P]
    const int* seq_start;     // [B + 1]
    const int* seq_slot;      // [B]
    float* out;               // [T, H P]
    int H, P, N, G;
    float* rec;               // [chunks, H, N P]: a chunk's own sum, then the state it starts with (where rows are whole pieces
                              // of 8: 8 leading halves and then 8 remainders, bfloat16, in the place of 8 floats)
    float* decay;             // [chunks, H]: exp(c_end)
    float* sums;              // [chunks, H, 2 * 64]: c_t of the chunk's tokens, then their steps
};

__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// ------------------------------------------------------------------ token by token
constexpr int SCAN_THREADS = 128;
constexpr int SCAN_RG = 8;              // groups of rows; 16 threads take neighbouring columns
constexpr int SCAN_STAGE = 8;           // tokens in shared memory at a time

// A block owns 16 V columns of one head's S; a thread R consecutive rows of V columns, in registers.
template <typename TX, int V, int R>
__global__ void __launch_bounds__(SCAN_THREADS) ssd_scan_kernel(SsdParams p) {
    constexpr int COLS = 16 * V, ROWS = SCAN_RG * R;
    extern __shared__ __align__(16) float sm[];
    float* sb = sm;                                        // [STAGE][ROWS]
    float* sc = sb + SCAN_STAGE * ROWS;
    float* sx = sc + SCAN_STAGE * ROWS;                    // [STAGE][COLS]
    float* red = sx + SCAN_STAGE * COLS;                   // [STAGE][RG][COLS]
    float* sd = red + SCAN_STAGE * SCAN_RG * COLS;         // [STAGE] decays, then [STAGE] steps
    const int tid = threadIdx.x, cq = tid & 15, rg = tid >> 4;
    const int h = blockIdx.y, b = blockIdx.z, col0 = blockIdx.x * COLS, col = col0 + cq * V;
    const int N = p.N, P = p.P, g = h / (p.H / p.G), inner = p.H * P;
    llb_grid_dependency_sync();
    const int tok0 = p.seq_start[b], n = p.seq_start[b + 1] - tok0;
    if (n == 0) return;
    float* st = p.state + ((size_t)p.seq_slot[b] * p.H + h) * N * P;
    float S[R][V];
#pragma unroll
    for (int m = 0; m < R; ++m) {
        const int i = rg * R + m;
#pragma unroll
        for (int e = 0; e < V; ++e) S[m][e] = 0.f;
        if (i < N && col < P) {
            if constexpr (V == 4) {
                const float4 q = *reinterpret_cast<const float4*>(st + (size_t)i * P + col);
                S[m][0] = q.x; S[m][1] = q.y; S[m][2] = q.z; S[m][3] = q.w;
            } else S[m][0] = st[(size_t)i * P + col];
        }
    }
    const float rate = -expf(p.a_log[h]), bias = p.dt_bias[h], skip = p.skip[h];
    for (int t0 = 0; t0 < n; t0 += SCAN_STAGE) {
        const int nt = min(SCAN_STAGE, n - t0);
        const TX* src = (const TX*)p.xbc + (size_t)(tok0 + t0) * p.ld;
        __syncthreads();
        for (int i = tid; i < nt * ROWS; i += SCAN_THREADS) {
            const int t = i / ROWS, r = i - t * ROWS;
            const TX* bc = src + (size_t)t * p.ld + inner + g * N + r;
            sb[i] = r < N ? to_f32(bc[0]) : 0.f;
            sc[i] = r < N ? to_f32(bc[p.G * N]) : 0.f;
        }
        for (int i = tid; i < nt * COLS; i += SCAN_THREADS) {
            const int t = i / COLS, c = col0 + i - t * COLS;
            sx[i] = c < P ? to_f32(src[(size_t)t * p.ld + h * P + c]) : 0.f;
        }
        if (tid < nt) {
            const float dt = softplus(p.dt[(size_t)(tok0 + t0 + tid) * p.dt_ld + h] + bias);
            sd[tid] = expf(rate * dt);
            sd[SCAN_STAGE + tid] = dt;
        }
        __syncthreads();
        for (int t = 0; t < nt; ++t) {
            const float a = sd[t], dt = sd[SCAN_STAGE + t];
            const float4* b4 = reinterpret_cast<const float4*>(sb + t * ROWS + rg * R);
            const float4* c4 = reinterpret_cast<const float4*>(sc + t * ROWS + rg * R);
            float x[V], y[V];
#pragma unroll
            for (int e = 0; e < V; ++e) {
                x[e] = dt * sx[t * COLS + cq * V + e];
                y[e] = 0.f;
            }
#pragma unroll
            for (int m = 0; m < R; m += 4) {
                const float4 bq = b4[m / 4], cq4 = c4[m / 4];
                const float bv[4] = {bq.x, bq.y, bq.z, bq.w}, cv[4] = {cq4.x, cq4.y, cq4.z, cq4.w};
#pragma unroll
                for (int k = 0; k < 4; ++k)
#pragma unroll
                    for (int e = 0; e < V; ++e) {
                        S[m + k][e] = fmaf(S[m + k][e], a, bv[k] * x[e]);
                        y[e] = fmaf(S[m + k][e], cv[k], y[e]);
                    }
            }
            float* r = red + (t * SCAN_RG + rg) * COLS + cq * V;
#pragma unroll
            for (int e = 0; e < V; ++e) r[e] = y[e];
        }
        __syncthreads();
        for (int i = tid; i < nt * COLS; i += SCAN_THREADS) {
            const int t = i / COLS, c = i - t * COLS;
            if (col0 + c >= P) continue;
            float y = 0.f;
#pragma unroll
            for (int k = 0; k < SCAN_RG; ++k) y += red[(t * SCAN_RG + k) * COLS + c];
            p.out[(size_t)(tok0 + t0 + t) * inner + h * P + col0 + c] = fmaf(skip, sx[i], y);
        }
    }
#pragma unroll
    for (int m = 0; m < R; ++m) {
        const int i = rg * R + m;
        if (i < N && col < P) {
            if constexpr (V == 4) *reinterpret_cast<float4*>(st + (size_t)i * P + col) = make_float4(S[m][0], S[m][1], S[m][2], S[m][3]);
            else st[(size_t)i * P + col] = S[m][0];
        }
    }
}

// ------------------------------------------------------------------ long steps, chunk by chunk
constexpr int CHUNK = 64;
constexpr int CHUNK_THREADS = 128;
static_assert(CHUNK_THREADS == 2 * CHUNK, "a thread per number of a chunk's sums");
constexpr int PT = 64;                  // value channels of a block
constexpr int PLD = PT + 8;             // row stride of a tile of PT columns: rows 16 bytes apart modulo 128

// The first chunk's place among all chunks of the step: sequences need not start at multiples of 64, and two never collide.
__device__ __forceinline__ int chunk_base(int tok0, int b) { return tok0 / CHUNK + b; }

__device__ __forceinline__ uint32_t smem_addr(const void* ptr) { return (uint32_t)__cvta_generic_to_shared(ptr); }
__device__ __forceinline__ void ldsm(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm_t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Two floats as two pairs of bfloat16: v = hi + lo up to 2^-17 of it.
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}

// 16 bytes into shared memory without waiting for them (zeros unless `in`).
__device__ __forceinline__ void copy16(bf16* dst, const bf16* src, bool in) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(in ? 16 : 0) : "memory");
}
__device__ __forceinline__ void copies_done() { asm volatile("cp.async.wait_all;" ::: "memory"); }

// [CHUNK rows, cols] of the operand into a tile of `pad` columns (a multiple of 16): 16-byte asynchronous copies where the rows
// allow it; zeros beyond `cols` and beyond the chunk's tokens.
template <int THREADS>
__device__ __forceinline__ void load_tile(bf16* dst, int dst_ld, const bf16* src, int ld, int rows, int cols, int pad, bool vec) {
    const int tid = threadIdx.x;
    if (vec) {                                             // 16 threads a row
        const int sub = (tid & 15) * 8;
#pragma unroll
        for (int k = 0; k < CHUNK * 16 / THREADS; ++k) {
            const int r = (tid >> 4) + k * (THREADS / 16);
            const bf16* row = src + (size_t)r * ld;
            for (int c = sub; c < pad; c += 128) copy16(dst + r * dst_ld + c, r < rows && c < cols ? row + c : src, r < rows && c < cols);
        }
    } else {
        for (int i = tid; i < CHUNK * pad; i += THREADS) {
            const int r = i / pad, c = i - r * pad;
            dst[r * dst_ld + c] = (r < rows && c < cols) ? src[(size_t)r * ld + c] : __float2bfloat16_rn(0.f);
        }
    }
}

// The first warp: step sizes and running log decays of the chunk's tokens (two a lane); tokens past its end repeat the last sum.
__device__ __forceinline__ void chunk_decays(const SsdParams& p, int row0, int nc, int h, float* scum, float* sdt) {
    const int lane = threadIdx.x;
    if (lane >= 32) return;
    const float rate = -expf(p.a_log[h]), bias = p.dt_bias[h];
    float dt[2], c[2];
#pragma unroll
    for (int k = 0; k < 2; ++k) {
        const int t = lane * 2 + k;
        dt[k] = t < nc ? softplus(p.dt[(size_t)(row0 + t) * p.dt_ld + h] + bias) : 0.f;
        c[k] = rate * dt[k];
    }
    c[1] += c[0];
    float sum = c[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const float other = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += other;
    }
    const float below = __shfl_up_sync(0xffffffffu, sum, 1);           // (not sum - c[1]: no difference of large sums)
    scum[lane * 2] = (lane ? below : 0.f) + c[0];
    scum[lane * 2 + 1] = sum;
    sdt[lane * 2] = dt[0];
    sdt[lane * 2 + 1] = dt[1];
}

// dS [N, PT columns] of one chunk of one head: the rows of B as the (transposed) A operand, w_s x_s as the B operand.
__global__ void __launch_bounds__(CHUNK_THREADS) ssd_chunk_state_kernel(SsdParams p, int npad, int ptiles, int vec) {
    extern __shared__ __align__(16) unsigned char raw[];
    const int bld = npad + 8;
    bf16* sB = reinterpret_cast<bf16*>(raw);               // [CHUNK][bld]
    bf16* sHi = sB + CHUNK * bld;                          // [CHUNK][PLD]
    bf16* sLo = sHi + CHUNK * PLD;
    __shared__ float scum[CHUNK], sdt[CHUNK];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, a4 = lane & 3;
    const int h = blockIdx.y / ptiles, p0 = (blockIdx.y - h * ptiles) * PT, b = blockIdx.z, c = blockIdx.x;
    const int N = p.N, P = p.P, g = h / (p.H / p.G), inner = p.H * P;
    llb_grid_dependency_sync();
    const int tok0 = p.seq_start[b], n = p.seq_start[b + 1] - tok0;
    if (c * CHUNK >= n) return;
    const int nc = min(CHUNK, n - c * CHUNK), row0 = tok0 + c * CHUNK;
    const bf16* src = (const bf16*)p.xbc + (size_t)row0 * p.ld;
    load_tile<CHUNK_THREADS>(sB, bld, src + inner + g * N, p.ld, nc, N, npad, vec);
    // (the rows of x are under way before the decays are formed)
    constexpr int XP = CHUNK * (PT / 8) / CHUNK_THREADS;
    uint4 xq[XP];
    if (vec) {
#pragma unroll
        for (int k = 0; k < XP; ++k) {
            const int i = tid + k * CHUNK_THREADS, r = i / (PT / 8), cc = (i - r * (PT / 8)) * 8;
            xq[k] = make_uint4(0u, 0u, 0u, 0u);
            if (r < nc && p0 + cc < P) xq[k] = *reinterpret_cast<const uint4*>(src + h * P + p0 + (size_t)r * p.ld + cc);
        }
    }
    chunk_decays(p, row0, nc, h, scum, sdt);
    __syncthreads();
    const float end = scum[CHUNK - 1];
    const size_t chunk = (size_t)(chunk_base(tok0, b) + c) * p.H + h;
    if (tid == 0 && p0 == 0) p.decay[chunk] = expf(end);
    if (p0 == 0) p.sums[chunk * 2 * CHUNK + tid] = tid < CHUNK ? scum[tid] : sdt[tid - CHUNK];
    {
        const bf16* xs = src + h * P + p0;
        if (vec) {
#pragma unroll
            for (int k = 0; k < XP; ++k) {
                const int i = tid + k * CHUNK_THREADS, r = i / (PT / 8), cc = (i - r * (PT / 8)) * 8;
                uint4 hi, lo;
                const float w = expf(end - scum[r]) * sdt[r];
                const __nv_bfloat162* x2 = reinterpret_cast<const __nv_bfloat162*>(&xq[k]);
                uint32_t* h4 = reinterpret_cast<uint32_t*>(&hi);
                uint32_t* l4 = reinterpret_cast<uint32_t*>(&lo);
#pragma unroll
                for (int e = 0; e < 4; ++e) split2(w * __low2float(x2[e]), w * __high2float(x2[e]), h4[e], l4[e]);
                *reinterpret_cast<uint4*>(sHi + r * PLD + cc) = hi;
                *reinterpret_cast<uint4*>(sLo + r * PLD + cc) = lo;
            }
        } else {
            for (int i = tid; i < CHUNK * PT; i += CHUNK_THREADS) {
                const int r = i / PT, cc = i - r * PT;
                const float v = (r < nc && p0 + cc < P) ? expf(end - scum[r]) * sdt[r] * to_f32(xs[(size_t)r * p.ld + cc]) : 0.f;
                const bf16 hi = __float2bfloat16_rn(v);
                sHi[r * PLD + cc] = hi;
                sLo[r * PLD + cc] = __float2bfloat16_rn(v - __bfloat162float(hi));
            }
        }
    }
    copies_done();
    __syncthreads();
    float* rec = p.rec + chunk * N * P;
    const uint32_t ab = smem_addr(sB) + (((lane & 7) + ((lane >> 4) << 3)) * bld + ((lane >> 3) & 1) * 8) * 2;
    const uint32_t xoff = ((lane & 15) * PLD + (lane >> 4) * 8) * 2;
    const uint32_t hb = smem_addr(sHi) + xoff, lb = smem_addr(sLo) + xoff;
    constexpr int MSTEP = CHUNK_THREADS / 32 * 16;         // a warp takes two tiles of 16 rows, this far apart, for every tile of x it loads
    for (int m0 = warp * 16; m0 < npad; m0 += 2 * MSTEP) {
        const bool two = m0 + MSTEP < npad;
        float acc[2][PT / 8][4];
#pragma unroll
        for (int m = 0; m < 2; ++m)
#pragma unroll
            for (int j = 0; j < PT / 8; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) acc[m][j][e] = 0.f;
#pragma unroll
        for (int k0 = 0; k0 < CHUNK; k0 += 16) {
            uint32_t a[2][4];
            ldsm_t(a[0], ab + (k0 * bld + m0) * 2);
            if (two) ldsm_t(a[1], ab + (k0 * bld + m0 + MSTEP) * 2);
#pragma unroll
            for (int j = 0; j < PT / 16; ++j) {
                uint32_t x[4], y[4];
                ldsm_t(x, hb + (k0 * PLD + j * 16) * 2);
                ldsm_t(y, lb + (k0 * PLD + j * 16) * 2);
#pragma unroll
                for (int m = 0; m < 2; ++m) {
                    if (m && !two) break;
                    mma(acc[m][2 * j], a[m], x[0], x[1]);
                    mma(acc[m][2 * j + 1], a[m], x[2], x[3]);
                    mma(acc[m][2 * j], a[m], y[0], y[1]);
                    mma(acc[m][2 * j + 1], a[m], y[2], y[3]);
                }
            }
        }
#pragma unroll
        for (int m = 0; m < 2; ++m) {
            if (m && !two) break;
#pragma unroll
            for (int j = 0; j < PT / 8; ++j)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int i = m0 + m * MSTEP + g8 + half * 8, cc = p0 + j * 8 + a4 * 2;
                    if (i >= N || cc >= P) continue;
                    float* dst = rec + (size_t)i * P + cc;
                    if (P % 2 == 0) *reinterpret_cast<float2*>(dst) = make_float2(acc[m][j][half * 2], acc[m][j][half * 2 + 1]);
                    else {
                        dst[0] = acc[m][j][half * 2];
                        if (cc + 1 < P) dst[1] = acc[m][j][half * 2 + 1];
                    }
                }
        }
    }
}

// rec of every chunk: its own sum in, the state it starts with out; the sequence's state is brought up to date.
template <int V>
__global__ void __launch_bounds__(128) ssd_chunk_prefix_kernel(SsdParams p) {
    constexpr int AHEAD = V == 8 ? 4 : 8;
    const int h = blockIdx.y, b = blockIdx.z, n_el = p.N * p.P, e0 = (blockIdx.x * 128 + threadIdx.x) * V;
    llb_grid_dependency_sync();
    const int tok0 = p.seq_start[b], n = p.seq_start[b + 1] - tok0, nc = (n + CHUNK - 1) / CHUNK;
    if (e0 >= n_el || nc == 0) return;
    float* st = p.state + ((size_t)p.seq_slot[b] * p.H + h) * n_el + e0;
    const size_t first = (size_t)chunk_base(tok0, b) * p.H + h, step = (size_t)p.H * n_el;
    float* rec = p.rec + first * n_el + e0;
    const float* dec = p.decay + first;
    float S[V];
    auto load = [&](float (&v)[V], const float* src) {
        if constexpr (V == 8) {
            const float4 q = reinterpret_cast<const float4*>(src)[0], r = reinterpret_cast<const float4*>(src)[1];
            v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w; v[4] = r.x; v[5] = r.y; v[6] = r.z; v[7] = r.w;
        } else v[0] = src[0];
    };
    auto store = [&](float* dst, const float (&v)[V]) {
        if constexpr (V == 8) {
            reinterpret_cast<float4*>(dst)[0] = make_float4(v[0], v[1], v[2], v[3]);
            reinterpret_cast<float4*>(dst)[1] = make_float4(v[4], v[5], v[6], v[7]);
        } else dst[0] = v[0];
    };
    auto store_start = [&](float* dst, const float (&v)[V]) {
        if constexpr (V == 8) {
            uint4 hi, lo;
            split2(v[0], v[1], hi.x, lo.x);
            split2(v[2], v[3], hi.y, lo.y);
            split2(v[4], v[5], hi.z, lo.z);
            split2(v[6], v[7], hi.w, lo.w);
            reinterpret_cast<uint4*>(dst)[0] = hi;
            reinterpret_cast<uint4*>(dst)[1] = lo;
        } else dst[0] = v[0];
    };
    load(S, st);
    for (int c0 = 0; c0 < nc; c0 += AHEAD) {
        float d[AHEAD][V], a[AHEAD];
#pragma unroll
        for (int k = 0; k < AHEAD; ++k)
            if (c0 + k < nc) {
                load(d[k], rec + (size_t)(c0 + k) * step);
                a[k] = dec[(size_t)(c0 + k) * p.H];
            }
#pragma unroll
        for (int k = 0; k < AHEAD; ++k)
            if (c0 + k < nc) {
                store_start(rec + (size_t)(c0 + k) * step, S);
#pragma unroll
                for (int e = 0; e < V; ++e) S[e] = fmaf(a[k], S[e], d[k][e]);
            }
    }
    store(st, S);
}

// y of one chunk of one head, PT columns: a warp takes 16 tokens and half of the columns (both halves' warps form the scores: that
// costs a quarter more products and doubles the warps that an SM's shared memory has room for).
constexpr int OUT_THREADS = 256, OUT_COLS = PT / 2;
__global__ void __launch_bounds__(OUT_THREADS) ssd_chunk_out_kernel(SsdParams p, int npad, int ptiles, int vec) {
    extern __shared__ __align__(16) unsigned char raw[];
    const int bld = npad + 8;
    bf16* sC = reinterpret_cast<bf16*>(raw);               // [CHUNK][bld]
    bf16* sB = sC + CHUNK * bld;                           // [CHUNK][bld]
    bf16* sX = sB + CHUNK * bld;                           // [CHUNK][PLD]
    bf16* sHi = sX + CHUNK * PLD;                          // [npad][PLD]: S_0
    bf16* sLo = sHi + npad * PLD;
    __shared__ float sums[2 * CHUNK];
    const float* scum = sums;
    const float* sdt = sums + CHUNK;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, a4 = lane & 3;
    const int h = blockIdx.y / ptiles, p0 = (blockIdx.y - h * ptiles) * PT, b = blockIdx.z, c = blockIdx.x;
    const int N = p.N, P = p.P, g = h / (p.H / p.G), inner = p.H * P;
    llb_grid_dependency_sync();
    const int tok0 = p.seq_start[b], n = p.seq_start[b + 1] - tok0;
    if (c * CHUNK >= n) return;
    const int nc = min(CHUNK, n - c * CHUNK), row0 = tok0 + c * CHUNK;
    const bf16* src = (const bf16*)p.xbc + (size_t)row0 * p.ld;
    const size_t chunk = (size_t)(chunk_base(tok0, b) + c) * p.H + h;
    const float my_sum = tid < 2 * CHUNK ? p.sums[chunk * 2 * CHUNK + tid] : 0.f;
    load_tile<OUT_THREADS>(sC, bld, src + inner + (p.G + g) * N, p.ld, nc, N, npad, vec);
    load_tile<OUT_THREADS>(sB, bld, src + inner + g * N, p.ld, nc, N, npad, vec);
    load_tile<OUT_THREADS>(sX, PLD, src + h * P + p0, p.ld, nc, min(PT, P - p0), PT, vec);
    {
        const float* rec = p.rec + chunk * N * P + p0;
        if (vec) {
            for (int i = tid; i < npad * (PT / 8); i += OUT_THREADS) {
                const int r = i / (PT / 8), cc = (i - r * (PT / 8)) * 8;
                const bool in = r < N && p0 + cc < P;
                const bf16* piece = reinterpret_cast<const bf16*>(in ? rec + (size_t)r * P + cc : rec);
                copy16(sHi + r * PLD + cc, piece, in);
                copy16(sLo + r * PLD + cc, piece + 8, in);
            }
        } else {
            for (int i = tid; i < npad * PT; i += OUT_THREADS) {
                const int r = i / PT, cc = i - r * PT;
                const float v = (r < N && p0 + cc < P) ? rec[(size_t)r * P + cc] : 0.f;
                const bf16 hi = __float2bfloat16_rn(v);
                sHi[r * PLD + cc] = hi;
                sLo[r * PLD + cc] = __float2bfloat16_rn(v - __bfloat162float(hi));
            }
        }
    }
    if (tid < 2 * CHUNK) sums[tid] = my_sum;
    copies_done();
    __syncthreads();
    const int t0 = (warp & 3) * 16, col0 = (warp >> 2) * OUT_COLS;
    if (t0 >= nc || p0 + col0 >= P) return;                // (no barrier follows)
    const uint32_t ca = smem_addr(sC) + ((t0 + (lane & 15)) * bld + (lane >> 4) * 8) * 2;
    const uint32_t bb = smem_addr(sB) + (((lane & 7) + ((lane >> 4) << 3)) * bld + ((lane >> 3) & 1) * 8) * 2;
    const uint32_t xoff = ((lane & 15) * PLD + (lane >> 4) * 8 + col0) * 2;
    const uint32_t xb = smem_addr(sX) + xoff, hb = smem_addr(sHi) + xoff, lb = smem_addr(sLo) + xoff;
    float acc[OUT_COLS / 8][4];
#pragma unroll
    for (int j = 0; j < OUT_COLS / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
    // ---- what the chunk starts with
#pragma unroll 2
    for (int k0 = 0; k0 < npad; k0 += 16) {
        uint32_t a[4];
        ldsm(a, ca + k0 * 2);
#pragma unroll
        for (int j = 0; j < OUT_COLS / 16; ++j) {
            uint32_t s[4];
            ldsm_t(s, hb + (k0 * PLD + j * 16) * 2);
            mma(acc[2 * j], a, s[0], s[1]);
            mma(acc[2 * j + 1], a, s[2], s[3]);
            ldsm_t(s, lb + (k0 * PLD + j * 16) * 2);
            mma(acc[2 * j], a, s[0], s[1]);
            mma(acc[2 * j + 1], a, s[2], s[3]);
        }
    }
    const float ct[2] = {scum[t0 + g8], scum[t0 + g8 + 8]};
    const float et[2] = {expf(ct[0]), expf(ct[1])};
#pragma unroll
    for (int j = 0; j < OUT_COLS / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[j][e] *= et[e >> 1];
    // ---- the chunk's own tokens, 16 at a time
    for (int s0 = 0; s0 <= t0; s0 += 16) {
        float w[2][4];
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) w[j][e] = 0.f;
#pragma unroll 4
        for (int k0 = 0; k0 < npad; k0 += 16) {
            uint32_t a[4], s[4];
            ldsm(a, ca + k0 * 2);
            ldsm(s, bb + (s0 * bld + k0) * 2);
            mma(w[0], a, s[0], s[1]);
            mma(w[1], a, s[2], s[3]);
        }
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int s = s0 + j * 8 + a4 * 2 + (e & 1), t = t0 + g8 + (e >> 1) * 8;
                w[j][e] = s <= t ? w[j][e] * (__expf(ct[e >> 1] - scum[s]) * sdt[s]) : 0.f;
            }
        uint32_t hi[4], lo[4];
        split2(w[0][0], w[0][1], hi[0], lo[0]);
        split2(w[0][2], w[0][3], hi[1], lo[1]);
        split2(w[1][0], w[1][1], hi[2], lo[2]);
        split2(w[1][2], w[1][3], hi[3], lo[3]);
#pragma unroll
        for (int j = 0; j < OUT_COLS / 16; ++j) {
            uint32_t x[4];
            ldsm_t(x, xb + (s0 * PLD + j * 16) * 2);
            mma(acc[2 * j], hi, x[0], x[1]);
            mma(acc[2 * j + 1], hi, x[2], x[3]);
            mma(acc[2 * j], lo, x[0], x[1]);
            mma(acc[2 * j + 1], lo, x[2], x[3]);
        }
    }
    const float skip = p.skip[h];
#pragma unroll
    for (int j = 0; j < OUT_COLS / 8; ++j)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int t = t0 + g8 + half * 8, cl = col0 + j * 8 + a4 * 2, cc = p0 + cl;
            if (t >= nc || cc >= P) continue;
            float* dst = p.out + (size_t)(row0 + t) * inner + h * P + cc;
            const float y0 = fmaf(skip, __bfloat162float(sX[t * PLD + cl]), acc[j][half * 2]);
            const float y1 = fmaf(skip, __bfloat162float(sX[t * PLD + cl + 1]), acc[j][half * 2 + 1]);
            if (P % 2 == 0) *reinterpret_cast<float2*>(dst) = make_float2(y0, y1);
            else {
                dst[0] = y0;
                if (cc + 1 < P) dst[1] = y1;
            }
        }
}

int set_smem(const void* kernel, int& have, size_t smem) {
    if ((int)smem <= have) return 0;
    if (smem > 227 * 1024) return (int)cudaErrorInvalidValue;
    if (smem > 40 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    have = (int)smem;
    return 0;
}

template <typename TX, int V, int R>
int launch_scan(const SsdParams& p, int B, cudaStream_t stream) {
    auto k = ssd_scan_kernel<TX, V, R>;
    constexpr int COLS = 16 * V, ROWS = SCAN_RG * R;
    constexpr size_t smem = (size_t)(SCAN_STAGE * (2 * ROWS + COLS + SCAN_RG * COLS) + 2 * SCAN_STAGE) * sizeof(float);
    static int have = 0;
    if (int rc = set_smem((const void*)k, have, smem)) return rc;
    llb_launch(k, dim3((p.P + COLS - 1) / COLS, p.H, B), dim3(SCAN_THREADS), smem, stream, p);
    return llb_status();
}
template <typename TX, int V>
int launch_scan_rows(const SsdParams& p, int B, cudaStream_t stream) {
    if (p.N <= 32) return launch_scan<TX, V, 4>(p, B, stream);
    if (p.N <= 64) return launch_scan<TX, V, 8>(p, B, stream);
    if (p.N <= 128) return launch_scan<TX, V, 16>(p, B, stream);
    return launch_scan<TX, V, 32>(p, B, stream);
}

bool sizes_ok(const SsdParams& p, int B) {
    return p.G > 0 && p.H > 0 && p.H % p.G == 0 && p.N > 0 && p.N <= 256 && p.P > 0 && p.H <= 65535 && B <= 65535 &&
           p.ld >= p.H * p.P + 2 * p.G * p.N;
}

// ------------------------------------------------------------------ gate and norm in parts
// TPR threads share a part of `size` channels; the gated values wait in shared memory for the part's root mean square.
template <typename TZ, typename TO, int TPR, int V>
__global__ void __launch_bounds__(256) gated_group_norm_kernel(const float* __restrict__ y, const TZ* __restrict__ z, int z_ld,
                                                               const float* __restrict__ w, TO* __restrict__ out, int parts, int groups,
                                                               int size, float eps) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[8];
    constexpr int ROWS = 256 / TPR;
    const int tid = threadIdx.x, l = tid % TPR, part = blockIdx.x * ROWS + tid / TPR;
    llb_grid_dependency_sync();
    const bool in = part < parts;
    const int t = part / groups, c0 = (part - t * groups) * size;
    float* row = sm + (tid / TPR) * size;
    float ss = 0.f;
    if (in) {
        const float* yr = y + (size_t)t * groups * size + c0;
        const TZ* zr = z + (size_t)t * z_ld + c0;
        for (int i = l * V; i < size; i += TPR * V) {
            float v[V], q[V];
            if constexpr (V == 4) {
                const float4 y4 = *reinterpret_cast<const float4*>(yr + i);
                v[0] = y4.x; v[1] = y4.y; v[2] = y4.z; v[3] = y4.w;
                if constexpr (sizeof(TZ) == 2) {
                    const uint2 z4 = *reinterpret_cast<const uint2*>(zr + i);
                    const bf16* zb = reinterpret_cast<const bf16*>(&z4);
#pragma unroll
                    for (int e = 0; e < 4; ++e) q[e] = to_f32(zb[e]);
                } else {
                    const float4 z4 = *reinterpret_cast<const float4*>(zr + i);
                    q[0] = z4.x; q[1] = z4.y; q[2] = z4.z; q[3] = z4.w;
                }
            } else {
                v[0] = yr[i];
                q[0] = to_f32(zr[i]);
            }
#pragma unroll
            for (int e = 0; e < V; ++e) {
                v[e] *= sizeof(TO) == 2 ? __fdividef(q[e], 1.0f + __expf(-q[e])) : q[e] / (1.0f + expf(-q[e]));
                ss = fmaf(v[e], v[e], ss);
                row[i + e] = v[e];
            }
        }
    }
    ss = warp_sum(ss);
    if constexpr (TPR > 32) {
        if ((tid & 31) == 0) red[tid >> 5] = ss;
        __syncthreads();
        ss = 0.f;
#pragma unroll
        for (int k = 0; k < 8; ++k) ss += red[k];
    }
    if (!in) return;
    const float inv = 1.0f / sqrtf(ss / (float)size + eps);
    TO* dst = out + (size_t)t * groups * size + c0;
    for (int i = l * V; i < size; i += TPR * V) {          // (a thread reads back what it wrote)
        if constexpr (V == 4) {
            const float4 w4 = *reinterpret_cast<const float4*>(w + c0 + i);
            const float wv[4] = {w4.x, w4.y, w4.z, w4.w};
            struct alignas(4 * sizeof(TO)) { TO v[4]; } q;
#pragma unroll
            for (int e = 0; e < 4; ++e) q.v[e] = from_f32<TO>(row[i + e] * inv * wv[e]);
            *reinterpret_cast<decltype(q)*>(dst + i) = q;
        } else dst[i] = from_f32<TO>(row[i] * inv * w[c0 + i]);
    }
}

}  // namespace

// The recurrence over the new tokens of every sequence, token by token.
LLB_API int llb_ssd_scan(SsdParams p, int x_dtype, int B, cudaStream_t stream) {
    if (B == 0) return 0;
    if (!sizes_ok(p, B)) return (int)cudaErrorInvalidValue;
    const bool vec = p.P % 4 == 0 && !((uintptr_t)p.state & 15);
    LLB_DISPATCH_DTYPE(x_dtype, TX, {
        return vec ? launch_scan_rows<TX, 4>(p, B, stream) : launch_scan_rows<TX, 1>(p, B, stream);
    });
    return (int)cudaErrorInvalidValue;
}

// Chunks of the step's scratch for T packed tokens of B sequences: p.rec holds chunks * H N P floats, p.decay chunks * H, p.sums
// chunks * H * 128.
LLB_API int llb_ssd_chunks(int T, int B) { return T / CHUNK + B + 1; }

// The same recurrence in chunks (bfloat16 operands).
LLB_API int llb_ssd_chunked(SsdParams p, int B, int max_new, cudaStream_t stream) {
    if (B == 0 || max_new == 0) return 0;
    const int npad = (p.N + 15) / 16 * 16, ptiles = (p.P + PT - 1) / PT, chunks = (max_new + CHUNK - 1) / CHUNK;
    if (!sizes_ok(p, B) || (long long)p.H * ptiles > 65535 || (((uintptr_t)p.rec | (uintptr_t)p.state | (uintptr_t)p.out) & 15))
        return (int)cudaErrorInvalidValue;
    const int vec = p.ld % 8 == 0 && p.P % 8 == 0 && p.N % 8 == 0 && !((uintptr_t)p.xbc & 15);
    const size_t tile = (size_t)CHUNK * (npad + 8) * 2, xt = (size_t)CHUNK * PLD * 2;
    {
        static int have = 0;
        const size_t smem = tile + 2 * xt;
        if (int rc = set_smem((const void*)ssd_chunk_state_kernel, have, smem)) return rc;
        llb_launch(ssd_chunk_state_kernel, dim3(chunks, p.H * ptiles, B), dim3(CHUNK_THREADS), smem, stream, p, npad, ptiles, vec);
        if (int rc = llb_status()) return rc;
    }
    if (vec) llb_launch(ssd_chunk_prefix_kernel<8>, dim3((p.N * p.P / 8 + 127) / 128, p.H, B), dim3(128), 0, stream, p);
    else llb_launch(ssd_chunk_prefix_kernel<1>, dim3((p.N * p.P + 127) / 128, p.H, B), dim3(128), 0, stream, p);
    if (int rc = llb_status()) return rc;
    {
        static int have = 0;
        const size_t smem = 2 * tile + xt + 2 * (size_t)npad * PLD * 2;
        if (int rc = set_smem((const void*)ssd_chunk_out_kernel, have, smem)) return rc;
        llb_launch(ssd_chunk_out_kernel, dim3(chunks, p.H * ptiles, B), dim3(OUT_THREADS), smem, stream, p, npad, ptiles, vec);
    }
    return llb_status();
}

LLB_API int llb_gated_group_norm(const float* y, const void* z, int z_dtype, int z_ld, const float* w, void* out, int out_dtype, int T,
                                 int groups, int size, float eps, cudaStream_t stream) {
    if (T == 0) return 0;
    if (groups < 1 || size < 1 || (size_t)size * 4 > 200 * 1024 || (long long)T * groups > 0x7fffffffll) return (int)cudaErrorInvalidValue;
    const int parts = T * groups;
    const bool vec = size % 4 == 0 && z_ld % 4 == 0 && !(((uintptr_t)y | (uintptr_t)z | (uintptr_t)w | (uintptr_t)out) & 15);
    const bool narrow = size <= 512;
    const size_t smem = (size_t)(narrow ? 8 : 1) * size * sizeof(float);
#define LLB_GGN(TPR, V)                                                                                                             \
    do {                                                                                                                            \
        auto k = gated_group_norm_kernel<TZ, TO, TPR, V>;                                                                           \
        static int have = 0;                                                                                                        \
        if (int rc = set_smem((const void*)k, have, smem)) return rc;                                                               \
        llb_launch(k, dim3((parts + 256 / TPR - 1) / (256 / TPR)), dim3(256), smem, stream, y, (const TZ*)z, z_ld, w, (TO*)out, parts, \
                   groups, size, eps);                                                                                              \
    } while (0)
    LLB_DISPATCH_DTYPE(z_dtype, TZ, {
        LLB_DISPATCH_DTYPE(out_dtype, TO, {
            if (narrow && vec) LLB_GGN(32, 4);
            else if (narrow) LLB_GGN(32, 1);
            else if (vec) LLB_GGN(256, 4);
            else LLB_GGN(256, 1);
        });
    });
#undef LLB_GGN
    return llb_status();
}
