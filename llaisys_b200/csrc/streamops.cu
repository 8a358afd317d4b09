// Passes over rows of the float32 residual stream for arrangements whose parts join the stream through a gate:
//
//   stream_join   v = x[r] + sigmoid(gate[r]) * delta[r] + rows_add[r] + vec_add        (each term optional; element by
//                 element; written back to x), then out[r] = v / sqrt(mean(v^2) + eps) * weight   (optional)
//   branch_mean   out[r] = mult * sum_b x_b[r] / sqrt(mean(x_b[r]^2) + eps) * w_b: several mixers' results, each normed
//                 over the row with a weight of its own, averaged
//   scale_rows    x *= c
//   softcap_rows  x <- c tanh(x / c)
//   layer_norm    out[r] = (v - mean(v)) / sqrt(mean((v - mean(v))^2) + eps) * weight, v = x[rows ? rows[r] : r]
//   copy_rows     rows of the stream, converted, into a matrix of another row stride
//
// One block (layer_norm of many rows: one to four warps) per row; a row is read once.
#include "common.cuh"

__device__ __forceinline__ float block_sum_256(float v, float* red) {
    v = warp_sum(v);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    __syncthreads();
    if (lane == 0) red[warp] = v;
    __syncthreads();
    float s = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) s += red[w];
    return s;
}

struct StreamJoinParams {
    float* x;                 // [T, H]
    const void* delta;        // [T, H] or null
    const float* gate;        // [T, ld_gate] logits or null (delta joins ungated)
    int ld_gate;
    const float* rows_add;    // [T, H] or null
    const float* vec_add;     // [H] or null
    const float* weight;      // [H] or null: no output
    void* out;                // [T, H]
    int H;
    float eps;
};

template <typename TD, typename TO>
__global__ void __launch_bounds__(256) stream_join_kernel(StreamJoinParams p) {
    extern __shared__ __align__(16) float row[];
    __shared__ float red[8];
    const int r = blockIdx.x, H = p.H;
    llb_grid_dependency_sync();
    float* x = p.x + (size_t)r * H;
    const TD* delta = p.delta ? (const TD*)p.delta + (size_t)r * H : nullptr;
    const float* gate = p.gate ? p.gate + (size_t)r * p.ld_gate : nullptr;
    const float* ra = p.rows_add ? p.rows_add + (size_t)r * H : nullptr;
    const float* va = p.vec_add;
    const bool write = delta || ra || va;
    float ss = 0.f;
    // four elements a thread and round where the row allows it (16-byte pieces of the float32 operands)
    const bool vec = H % 4 == 0 && p.ld_gate % 4 == 0 &&
                     !(((uintptr_t)p.x | (uintptr_t)p.delta | (uintptr_t)p.gate | (uintptr_t)p.rows_add | (uintptr_t)p.vec_add) & 15);
    if (vec) {
        for (int i = threadIdx.x * 4; i < H; i += 1024) {
            float4 v = *reinterpret_cast<const float4*>(x + i);
            float* e = reinterpret_cast<float*>(&v);
            if (ra) {
                const float4 a = *reinterpret_cast<const float4*>(ra + i);
                e[0] += a.x; e[1] += a.y; e[2] += a.z; e[3] += a.w;
            }
            if (va) {
                const float4 a = *reinterpret_cast<const float4*>(va + i);
                e[0] += a.x; e[1] += a.y; e[2] += a.z; e[3] += a.w;
            }
            if (delta) {
                float d[4];
#pragma unroll
                for (int u = 0; u < 4; ++u) d[u] = to_f32(delta[i + u]);
                if (gate) {
                    const float4 g = *reinterpret_cast<const float4*>(gate + i);
                    const float gg[4] = {g.x, g.y, g.z, g.w};
#pragma unroll
                    for (int u = 0; u < 4; ++u) d[u] = d[u] / (1.0f + expf(-gg[u]));
                }
#pragma unroll
                for (int u = 0; u < 4; ++u) e[u] += d[u];
            }
            if (write) *reinterpret_cast<float4*>(x + i) = v;
            *reinterpret_cast<float4*>(row + i) = v;
            ss += (e[0] * e[0] + e[1] * e[1]) + (e[2] * e[2] + e[3] * e[3]);
        }
    } else {
        for (int i = threadIdx.x; i < H; i += 256) {
            float v = x[i];
            if (ra) v += ra[i];
            if (va) v += va[i];
            if (delta) {
                const float dl = to_f32(delta[i]);
                v += gate ? dl / (1.0f + expf(-gate[i])) : dl;
            }
            if (write) x[i] = v;
            row[i] = v;
            ss = fmaf(v, v, ss);
        }
    }
    if (!p.weight) return;
    ss = block_sum_256(ss, red);
    const float inv = 1.0f / sqrtf(ss / (float)H + p.eps);
    const float* w = p.weight;
    TO* out = (TO*)p.out + (size_t)r * H;
    for (int i = threadIdx.x; i < H; i += 256) out[i] = from_f32<TO>(row[i] * inv * w[i]);
}

LLB_API int llb_stream_join(StreamJoinParams p, int delta_dtype, int out_dtype, int T, cudaStream_t stream) {
    if (T == 0) return 0;
    const size_t smem = (size_t)p.H * sizeof(float);
    if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
    LLB_DISPATCH_DTYPE(delta_dtype, TD, {
        LLB_DISPATCH_DTYPE(out_dtype, TO, {
            auto k = stream_join_kernel<TD, TO>;
            static bool configured = false;
            if (!configured && smem > 48 * 1024) {
                cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
                if (e != cudaSuccess) return (int)e;
                configured = true;
            }
            llb_launch(k, dim3(T), dim3(256), smem, stream, p);
        });
    });
    return llb_status();
}

// ------------------------------------------------------------------ mean of normed branches
struct BranchMeanParams {
    const float* x[4];        // [T, H] each
    const void* w[4];         // [H] each
    int n;
    float* out;               // [T, H]
    int H;
    float eps, mult;
};

template <typename TW>
__global__ void __launch_bounds__(256) branch_mean_kernel(BranchMeanParams p) {
    __shared__ float red[8];
    const int r = blockIdx.x, H = p.H;
    llb_grid_dependency_sync();
    float inv[4];
    for (int b = 0; b < p.n; ++b) {
        const float* x = p.x[b] + (size_t)r * H;
        float ss = 0.f;
        for (int i = threadIdx.x; i < H; i += 256) ss = fmaf(x[i], x[i], ss);
        ss = block_sum_256(ss, red);
        inv[b] = 1.0f / sqrtf(ss / (float)H + p.eps);
    }
    for (int i = threadIdx.x; i < H; i += 256) {
        float acc = 0.f;
        for (int b = 0; b < p.n; ++b) acc += p.x[b][(size_t)r * H + i] * inv[b] * to_f32(((const TW*)p.w[b])[i]);
        p.out[(size_t)r * H + i] = acc * p.mult;
    }
}

LLB_API int llb_branch_mean(BranchMeanParams p, int w_dtype, int T, cudaStream_t stream) {
    if (T == 0) return 0;
    if (p.n < 1 || p.n > 4) return (int)cudaErrorInvalidValue;
    LLB_DISPATCH_DTYPE(w_dtype, TW, llb_launch(branch_mean_kernel<TW>, dim3(T), dim3(256), 0, stream, p));
    return llb_status();
}

// ------------------------------------------------------------------ layer norm
// The mean first, then the squares of the deviations from it, both over the row in registers (or, for widths that are no
// multiple of 4 or beyond 16,384, in shared memory).  TPR threads share a row; a thread holds PER pieces of 16 bytes.
template <int TPR>
__device__ __forceinline__ float row_sum(float v, float* red) {
    v = warp_sum(v);
    if (TPR == 32) return v;
    constexpr int W = TPR / 32;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, first = warp / W * W;
    __syncthreads();
    if (lane == 0) red[warp] = v;
    __syncthreads();
    float s = 0.f;
#pragma unroll
    for (int w = 0; w < W; ++w) s += red[first + w];
    return s;
}

template <typename TW, typename TO, int TPR, int PER>
__global__ void __launch_bounds__(256) layer_norm_kernel(const float* __restrict__ x, const TW* __restrict__ weight, TO* __restrict__ out,
                                                         const int* __restrict__ rows, int R, int H, float eps) {
    __shared__ float red[8];
    const int tid = threadIdx.x % TPR, r = blockIdx.x * (256 / TPR) + threadIdx.x / TPR;
    llb_grid_dependency_sync();
    const bool live = r < R;                               // (threads past the end take part in the barriers)
    const float* src = x + (size_t)(rows ? rows[live ? r : 0] : (live ? r : 0)) * H;
    float4 v[PER];
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int j = (tid + i * TPR) * 4;
        v[i] = j < H ? *reinterpret_cast<const float4*>(src + j) : make_float4(0.f, 0.f, 0.f, 0.f);
        s += (v[i].x + v[i].y) + (v[i].z + v[i].w);
    }
    const float mean = row_sum<TPR>(s, red) / (float)H;
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        if ((tid + i * TPR) * 4 >= H) continue;
        v[i].x -= mean;
        v[i].y -= mean;
        v[i].z -= mean;
        v[i].w -= mean;
        ss += (v[i].x * v[i].x + v[i].y * v[i].y) + (v[i].z * v[i].z + v[i].w * v[i].w);
    }
    const float inv = 1.0f / sqrtf(row_sum<TPR>(ss, red) / (float)H + eps);
    TO* dst = out + (size_t)r * H;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int j = (tid + i * TPR) * 4;
        if (j >= H || !live) continue;
        const float y[4] = {v[i].x, v[i].y, v[i].z, v[i].w};
        alignas(16) TO o[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) o[e] = from_f32<TO>(y[e] * inv * to_f32(weight[j + e]));
        if constexpr (sizeof(TO) == 4) *reinterpret_cast<float4*>(dst + j) = *reinterpret_cast<const float4*>(o);
        else *reinterpret_cast<uint2*>(dst + j) = *reinterpret_cast<const uint2*>(o);
    }
}

template <typename TW, typename TO>
__global__ void __launch_bounds__(256) layer_norm_any_kernel(const float* __restrict__ x, const TW* __restrict__ weight, TO* __restrict__ out,
                                                             const int* __restrict__ rows, int H, float eps) {
    extern __shared__ __align__(16) float row[];
    __shared__ float red[8];
    const int r = blockIdx.x;
    llb_grid_dependency_sync();
    const float* src = x + (size_t)(rows ? rows[r] : r) * H;
    float s = 0.f;
    for (int i = threadIdx.x; i < H; i += 256) s += row[i] = src[i];
    const float mean = block_sum_256(s, red) / (float)H;
    float ss = 0.f;
    for (int i = threadIdx.x; i < H; i += 256) ss = fmaf(row[i] - mean, row[i] - mean, ss);
    const float inv = 1.0f / sqrtf(block_sum_256(ss, red) / (float)H + eps);
    for (int i = threadIdx.x; i < H; i += 256) out[(size_t)r * H + i] = from_f32<TO>((row[i] - mean) * inv * to_f32(weight[i]));
}

template <typename TW, typename TO>
static int layer_norm_launch(const float* x, const TW* w, TO* out, const int* rows, int R, int H, float eps, cudaStream_t stream) {
    if (H % 4 == 0 && H <= 16384 && !(((uintptr_t)x | (uintptr_t)out) & 15)) {
#define LLB_LN(TPR, PER) do { llb_launch(layer_norm_kernel<TW, TO, TPR, PER>, dim3((R + 256 / TPR - 1) / (256 / TPR)), dim3(256), 0,     \
                                         stream, x, w, out, rows, R, H, eps); return llb_status(); } while (0)
        if (R >= 256) {                                    // many rows: a warp, or four, per row
            if (H <= 512) LLB_LN(32, 4);
            if (H <= 1024) LLB_LN(128, 2);
            if (H <= 1536) LLB_LN(128, 3);
            if (H <= 2048) LLB_LN(128, 4);
            if (H <= 4096) LLB_LN(128, 8);
        }
        if (H <= 1024) LLB_LN(256, 1);
        if (H <= 2048) LLB_LN(256, 2);
        if (H <= 4096) LLB_LN(256, 4);
        LLB_LN(256, 16);
#undef LLB_LN
    }
    const size_t smem = (size_t)H * sizeof(float);
    if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
    auto k = layer_norm_any_kernel<TW, TO>;
    static bool configured = false;
    if (!configured && smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    llb_launch(k, dim3(R), dim3(256), smem, stream, x, w, out, rows, H, eps);
    return llb_status();
}

LLB_API int llb_layer_norm(const float* x, const void* weight, int w_dtype, void* out, int out_dtype, const int* rows, int R, int H,
                           float eps, cudaStream_t stream) {
    if (R == 0) return 0;
    LLB_DISPATCH_DTYPE(w_dtype, TW, {
        LLB_DISPATCH_DTYPE(out_dtype, TO, { return layer_norm_launch<TW, TO>(x, (const TW*)weight, (TO*)out, rows, R, H, eps, stream); });
    });
    return 0;
}

// ------------------------------------------------------------------ rows of the stream into another matrix
template <typename TO>
__global__ void __launch_bounds__(256) copy_rows_kernel(const float* __restrict__ x, TO* __restrict__ out, int ld, int H) {
    llb_grid_dependency_sync();
    const float* src = x + (size_t)blockIdx.x * H;
    TO* dst = out + (size_t)blockIdx.x * ld;
    const bool vec = H % 4 == 0 && ld % 4 == 0 && !(((uintptr_t)x | (uintptr_t)out) & 15);
    if (vec) {
        for (int i = threadIdx.x * 4; i < H; i += 1024) {
            const float4 v = *reinterpret_cast<const float4*>(src + i);
            alignas(16) TO o[4] = {from_f32<TO>(v.x), from_f32<TO>(v.y), from_f32<TO>(v.z), from_f32<TO>(v.w)};
            if constexpr (sizeof(TO) == 4) *reinterpret_cast<float4*>(dst + i) = *reinterpret_cast<const float4*>(o);
            else *reinterpret_cast<uint2*>(dst + i) = *reinterpret_cast<const uint2*>(o);
        }
        return;
    }
    for (int i = threadIdx.x; i < H; i += 256) dst[i] = from_f32<TO>(src[i]);
}

LLB_API int llb_copy_rows(const float* x, void* out, int out_dtype, int ld, int T, int H, cudaStream_t stream) {
    if (T == 0) return 0;
    LLB_DISPATCH_DTYPE(out_dtype, TO, llb_launch(copy_rows_kernel<TO>, dim3(T), dim3(256), 0, stream, x, (TO*)out, ld, H));
    return llb_status();
}

// ------------------------------------------------------------------ x *= c
__global__ void scale_rows_kernel(float* __restrict__ x, size_t n, float c) {
    llb_grid_dependency_sync();
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) x[i] *= c;
}

LLB_API int llb_scale_rows(float* x, long long n, float c, cudaStream_t stream) {
    if (n == 0) return 0;
    llb_launch(scale_rows_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, stream, x, (size_t)n, c);
    return llb_status();
}

__global__ void softcap_rows_kernel(float* __restrict__ x, size_t n, float c) {
    llb_grid_dependency_sync();
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) x[i] = c * tanhf(x[i] / c);
}

LLB_API int llb_softcap_rows(float* x, long long n, float c, cudaStream_t stream) {
    if (n == 0) return 0;
    llb_launch(softcap_rows_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, stream, x, (size_t)n, c);
    return llb_status();
}
