// Short causal convolutions over time, one filter per channel, whose last taps - 1 inputs are carried from step to step in a
// float32 state row per sequence (zeros when the sequence starts):
//
//     y_t[c] = bias[c] + sum_j w[j][c] u_(t - taps + 1 + j)[c]
//
//   short_conv   y, optionally through silu, into a matrix of its own
//   conv_heads   y of packed query and key heads, then what the attention needs of them: the values (a head's convolved key
//                before the rotation, times a constant), the rotation of the first `rot` dimensions of queries and keys
//                (pairs (i, i + rot/2)), and, when asked, the keys' and values' rows in the paged cache.  One pass, float32
//                arithmetic, one rounding.
//
// A thread takes a few channels of a run of consecutive tokens of one sequence.  A run is at least as long as the convolution
// reaches back, so only a sequence's first run reads the carried inputs; its threads leave the new ones.
#include "common.cuh"

namespace {

struct ShortConv {
    const void* x;            // [T, ld], the convolution's inputs
    int ld;
    const float* w;           // [taps, C], the last row for the current token
    const float* bias;        // [C] or null
    float* state;             // [slots, (taps - 1) C], oldest input first (null with one tap)
    const int* seq_start;     // [B + 1]
    const int* seq_slot;      // [B]
    int C, taps;
};

constexpr int RUN = 8;
constexpr int THREADS = 128;
__host__ __device__ constexpr int run_length(int taps) { return taps - 1 > RUN ? taps - 1 : RUN; }

template <typename T, int U> struct alignas(sizeof(T) * U) Piece { T v[U]; };

// The convolution of PIECES pieces of U neighbouring channels (columns col[i], where have[i]) over the tokens of the run that
// starts at token at0 of the sequence; emit(t, v) gets every token's results
// (with constant taps the loop over the run is unrolled, and t - at0 is a constant there).
template <typename T, int TAPS, int PIECES, int U, typename EMIT>
__device__ __forceinline__ void conv_run(const ShortConv& p, const int (&col)[PIECES], const bool (&have)[PIECES], int b, int tok0, int n,
                                         int at0, EMIT&& emit) {
    const int taps = TAPS > 0 ? TAPS : p.taps, back = taps - 1, hi = min(n, at0 + run_length(taps));
    const T* x = (const T*)p.x + (size_t)tok0 * p.ld;
    float* st = back > 0 ? p.state + (size_t)p.seq_slot[b] * back * p.C : nullptr;
    auto input = [&](float (&v)[PIECES][U], int r) {       // of token r of the sequence; r < 0: carried
#pragma unroll
        for (int i = 0; i < PIECES; ++i) {
#pragma unroll
            for (int e = 0; e < U; ++e) v[i][e] = 0.f;
            if (!have[i]) continue;
            if (r >= 0) {
                const Piece<T, U> q = *reinterpret_cast<const Piece<T, U>*>(x + (ptrdiff_t)r * p.ld + col[i]);
#pragma unroll
                for (int e = 0; e < U; ++e) v[i][e] = to_f32(q.v[e]);
            } else {
                const Piece<float, U> q = *reinterpret_cast<const Piece<float, U>*>(st + (size_t)(r + back) * p.C + col[i]);
#pragma unroll
                for (int e = 0; e < U; ++e) v[i][e] = q.v[e];
            }
        }
    };
    auto vec = [&](float (&v)[PIECES][U], const float* src) {
#pragma unroll
        for (int i = 0; i < PIECES; ++i) {
            Piece<float, U> q = {};
            if (have[i] && src) q = *reinterpret_cast<const Piece<float, U>*>(src + col[i]);
#pragma unroll
            for (int e = 0; e < U; ++e) v[i][e] = q.v[e];
        }
    };
    auto keep = [&](int j, const float (&v)[PIECES][U]) {
#pragma unroll
        for (int i = 0; i < PIECES; ++i)
            if (have[i]) {
                Piece<float, U> q;
#pragma unroll
                for (int e = 0; e < U; ++e) q.v[e] = v[i][e];
                *reinterpret_cast<Piece<float, U>*>(st + (size_t)j * p.C + col[i]) = q;
            }
    };
    float bias[PIECES][U];
    vec(bias, p.bias);
    if constexpr (TAPS > 0) {
        constexpr int BACK = TAPS - 1;
        float w[TAPS][PIECES][U], in[BACK + RUN][PIECES][U];
#pragma unroll
        for (int j = 0; j < BACK + RUN; ++j) {
            const int r = at0 - BACK + j;
            if (r < hi) input(in[j], r);
            else {
#pragma unroll
                for (int i = 0; i < PIECES; ++i)
#pragma unroll
                    for (int e = 0; e < U; ++e) in[j][i][e] = 0.f;
            }
        }
#pragma unroll
        for (int j = 0; j < TAPS; ++j) vec(w[j], p.w + (size_t)j * p.C);
#pragma unroll
        for (int u = 0; u < RUN; ++u) {
            if (at0 + u >= hi) break;
            float v[PIECES][U];
#pragma unroll
            for (int i = 0; i < PIECES; ++i)
#pragma unroll
                for (int e = 0; e < U; ++e) {
                    v[i][e] = bias[i][e];
#pragma unroll
                    for (int j = 0; j < TAPS; ++j) v[i][e] = fmaf(w[j][i][e], in[u + j][i][e], v[i][e]);
                }
            emit(at0 + u, v);
        }
        if (at0 == 0) {
#pragma unroll
            for (int j = 0; j < BACK; ++j) {               // the input of token n - BACK + j, ascending: nothing still needed is overwritten
                if (n == 1) keep(j, in[j + 1]);
                else {
                    float v[PIECES][U];
                    input(v, n - BACK + j);
                    keep(j, v);
                }
            }
        }
    } else {
        for (int t = at0; t < hi; ++t) {
            float v[PIECES][U], in[PIECES][U], w[PIECES][U];
#pragma unroll
            for (int i = 0; i < PIECES; ++i)
#pragma unroll
                for (int e = 0; e < U; ++e) v[i][e] = bias[i][e];
            for (int j = 0; j < taps; ++j) {
                input(in, t - back + j);
                vec(w, p.w + (size_t)j * p.C);
#pragma unroll
                for (int i = 0; i < PIECES; ++i)
#pragma unroll
                    for (int e = 0; e < U; ++e) v[i][e] = fmaf(w[i][e], in[i][e], v[i][e]);
            }
            emit(t, v);
        }
        if (at0 == 0)
            for (int j = 0; j < back; ++j) {               // ascending: what is still needed is not overwritten
                float v[PIECES][U];
                input(v, n - back + j);
                keep(j, v);
            }
    }
}

template <typename T, typename TO, int TAPS, int U>
__global__ void __launch_bounds__(THREADS) short_conv_kernel(ShortConv p, TO* __restrict__ out, int ldo, int silu) {
    const int b = blockIdx.z, at0 = blockIdx.y * run_length(TAPS > 0 ? TAPS : p.taps);
    const int tok0 = p.seq_start[b], n = p.seq_start[b + 1] - tok0;
    const int col[1] = {(int)(blockIdx.x * THREADS + threadIdx.x) * U};
    const bool have[1] = {col[0] < p.C};
    llb_grid_dependency_sync();
    if (at0 >= n || !have[0]) return;
    conv_run<T, TAPS, 1, U>(p, col, have, b, tok0, n, at0, [&](int t, float (&v)[1][U]) {
        Piece<TO, U> q;
#pragma unroll
        for (int e = 0; e < U; ++e) {
            float y = v[0][e];
            // (a result that is rounded to bfloat16 takes the special-function unit)
            if (silu) y = sizeof(TO) == 2 ? __fdividef(y, 1.0f + __expf(-y)) : y / (1.0f + expf(-y));
            q.v[e] = from_f32<TO>(y);
        }
        *reinterpret_cast<Piece<TO, U>*>(out + (size_t)(tok0 + t) * ldo + col[0]) = q;
    });
}

struct ConvHeads {
    ShortConv conv;           // x: n_q query heads of d channels, then n_k key heads
    void* out;                // [T, ldo]: queries, keys (both rotated), values (n_k heads of d)
    int ldo;
    int n_q, n_k, d, rot;
    float v_mult;
    const float* cos_t;       // [table_rows, rot / 2]
    const float* sin_t;
    int table_rows;
    const int* tok_pos;
    int append;
    const int* seq_len_before;
    void* kpool;
    void* vpool;
    const int* page_table;
    int table_stride, ring, pinned;
    int* err;
};

// A thread's two pieces are the two sides of U rotated pairs, or 2 U neighbours of a head's unrotated rest.
template <typename T, int TAPS, int U>
__global__ void __launch_bounds__(THREADS) conv_heads_kernel(ConvHeads p) {
    const int b = blockIdx.z, at0 = blockIdx.y * run_length(TAPS > 0 ? TAPS : p.conv.taps);
    const int tok0 = p.conv.seq_start[b], n = p.conv.seq_start[b + 1] - tok0;
    const int half = p.rot >> 1, turned = half / U, units = turned + (p.d - p.rot + 2 * U - 1) / (2 * U);
    const int id = blockIdx.x * THREADS + threadIdx.x, head = id / units, j = id - head * units;
    llb_grid_dependency_sync();
    if (at0 >= n || head >= p.n_q + p.n_k) return;
    const bool pair = j < turned, is_k = head >= p.n_q;
    const int first = pair ? j * U : p.rot + (j - turned) * 2 * U, second = pair ? first + half : first + U;
    const int col[2] = {head * p.d + first, head * p.d + second};
    const bool have[2] = {true, second < p.d};
    const int* table = p.append ? p.page_table + (size_t)b * p.table_stride : nullptr;
    const int last = p.append ? p.seq_len_before[b] + n - 1 : 0, kvh = head - p.n_q;
    T* kpool = (T*)p.kpool;
    T* vpool = (T*)p.vpool;
    const int pos0 = __ldg(p.tok_pos + tok0);              // (a sequence's tokens of a step stand at consecutive positions)
    if (p.rot > 0 && (pos0 < 0 || pos0 + n > p.table_rows)) {
        atomicExch(p.err, 2);
        return;
    }
    // what the run's tokens need beside their inputs is under way before the convolution waits for those: the angles, and where
    // the (at most two) pages of a short run's cache rows lie
    constexpr bool AHEAD = TAPS > 0;
    constexpr int NA = AHEAD ? RUN : 1;
    float ca[NA][U], sa[NA][U];
    const bool store_any = is_k && p.append;
    size_t page_at[2] = {0, 0};
    const int lp0 = (pos0 + at0) / LLB_PAGE;
    if constexpr (AHEAD) {
        if (pair)
#pragma unroll
            for (int u = 0; u < RUN; ++u)
#pragma unroll
                for (int e = 0; e < U; ++e) {
                    const bool in = at0 + u < n;
                    ca[u][e] = in ? __ldg(p.cos_t + (size_t)(pos0 + at0 + u) * half + first + e) : 1.f;
                    sa[u][e] = in ? __ldg(p.sin_t + (size_t)(pos0 + at0 + u) * half + first + e) : 0.f;
                }
        if (store_any) {
            const int lp1 = (pos0 + min(n, at0 + RUN) - 1) / LLB_PAGE;
            page_at[0] = paged_row(table, p.ring, lp0 * LLB_PAGE, kvh, p.n_k, p.d, p.pinned);
            page_at[1] = lp1 != lp0 ? paged_row(table, p.ring, lp1 * LLB_PAGE, kvh, p.n_k, p.d, p.pinned) : page_at[0];
        }
    }
    conv_run<T, TAPS, 2, U>(p.conv, col, have, b, tok0, n, at0, [&](int t, float (&v)[2][U]) {
        const int pos = pos0 + t;
        T* row = (T*)p.out + (size_t)(tok0 + t) * p.ldo;
        const bool store = store_any && paged_survives(pos / LLB_PAGE, last / LLB_PAGE, p.ring, p.pinned);
        const size_t at = !store ? 0 : AHEAD ? (pos / LLB_PAGE == lp0 ? page_at[0] : page_at[1]) + (size_t)(pos % LLB_PAGE) * p.d
                                             : paged_row(table, p.ring, pos, kvh, p.n_k, p.d, p.pinned);
        Piece<T, U> q[2];
        if (is_k) {
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                if (!have[i]) continue;
#pragma unroll
                for (int e = 0; e < U; ++e) q[i].v[e] = from_f32<T>(v[i][e] * p.v_mult);
                *reinterpret_cast<Piece<T, U>*>(row + (size_t)p.n_k * p.d + col[i]) = q[i];
                if (store) *reinterpret_cast<Piece<T, U>*>(vpool + at + col[i] - head * p.d) = q[i];
            }
        }
        if (pair) {
#pragma unroll
            for (int e = 0; e < U; ++e) {
                const float c = AHEAD ? ca[t - at0][e] : __ldg(p.cos_t + (size_t)pos * half + first + e);
                const float s = AHEAD ? sa[t - at0][e] : __ldg(p.sin_t + (size_t)pos * half + first + e);
                const float x0 = v[0][e], x1 = v[1][e];
                v[0][e] = x0 * c - x1 * s;
                v[1][e] = x1 * c + x0 * s;
            }
        }
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            if (!have[i]) continue;
#pragma unroll
            for (int e = 0; e < U; ++e) q[i].v[e] = from_f32<T>(v[i][e]);
            *reinterpret_cast<Piece<T, U>*>(row + col[i]) = q[i];
            if (store) *reinterpret_cast<Piece<T, U>*>(kpool + at + col[i] - head * p.d) = q[i];
        }
    });
}

bool aligned(const void* a, size_t bytes) { return ((uintptr_t)a & (bytes - 1)) == 0; }

bool conv_ok(const ShortConv& p, int B) { return p.C > 0 && p.taps >= 1 && p.ld >= p.C && B <= 65535 && (p.taps == 1 || p.state); }

}  // namespace

LLB_API int llb_short_conv(ShortConv p, int x_dtype, void* out, int out_dtype, int ldo, int silu, int B, int max_new, cudaStream_t stream) {
    if (B == 0 || max_new == 0) return 0;
    const int runs = (max_new + run_length(p.taps) - 1) / run_length(p.taps);
    if (!conv_ok(p, B) || ldo < p.C || runs > 65535) return (int)cudaErrorInvalidValue;
    const bool vec = p.C % 4 == 0 && p.ld % 4 == 0 && ldo % 4 == 0 && aligned(p.x, 16) && aligned(out, 16) && aligned(p.w, 16) &&
                     aligned(p.bias, 16) && aligned(p.state, 16);
    const int per = vec ? 4 : 1;
    const dim3 grid((p.C + THREADS * per - 1) / (THREADS * per), runs, B), block(THREADS);
#define LLB_SC(TAPS, U) llb_launch(short_conv_kernel<TX, TO, TAPS, U>, grid, block, 0, stream, p, (TO*)out, ldo, silu)
    LLB_DISPATCH_DTYPE(x_dtype, TX, {
        LLB_DISPATCH_DTYPE(out_dtype, TO, {
            if (vec && p.taps == 4) LLB_SC(4, 4);
            else if (vec) LLB_SC(0, 4);
            else if (p.taps == 4) LLB_SC(4, 1);
            else LLB_SC(0, 1);
        });
    });
#undef LLB_SC
    return llb_status();
}

LLB_API int llb_conv_heads(ConvHeads p, int dtype, int B, int max_new, cudaStream_t stream) {
    if (B == 0 || max_new == 0) return 0;
    const int runs = (max_new + run_length(p.conv.taps) - 1) / run_length(p.conv.taps);
    if (!conv_ok(p.conv, B) || runs > 65535 || p.n_q < 0 || p.n_k <= 0 || p.d <= 0 || p.rot < 0 || p.rot % 2 || p.rot > p.d ||
        p.conv.C != (p.n_q + p.n_k) * p.d || p.ldo < (p.n_q + 2 * p.n_k) * p.d)
        return (int)cudaErrorInvalidValue;
    const bool vec = p.d % 4 == 0 && p.rot % 4 == 0 && p.conv.ld % 2 == 0 && p.ldo % 2 == 0 && aligned(p.conv.x, 8) && aligned(p.out, 8) &&
                     aligned(p.conv.w, 8) && aligned(p.conv.bias, 8) && aligned(p.conv.state, 8) && aligned(p.kpool, 8) && aligned(p.vpool, 8);
    const int per = vec ? 2 : 1;
    const int units = (p.n_q + p.n_k) * (p.rot / 2 / per + (p.d - p.rot + 2 * per - 1) / (2 * per));
    const dim3 grid((units + THREADS - 1) / THREADS, runs, B), block(THREADS);
    LLB_DISPATCH_DTYPE(dtype, TT, {
        if (vec && p.conv.taps == 4) llb_launch(conv_heads_kernel<TT, 4, 2>, grid, block, 0, stream, p);
        else if (vec) llb_launch(conv_heads_kernel<TT, 0, 2>, grid, block, 0, stream, p);
        else if (p.conv.taps == 4) llb_launch(conv_heads_kernel<TT, 4, 1>, grid, block, 0, stream, p);
        else llb_launch(conv_heads_kernel<TT, 0, 1>, grid, block, 0, stream, p);
    });
    return llb_status();
}
