// What follows a recurrence: every head's result is RMS-normed over its value channels with a weight shared by the heads and
// multiplied by an output gate, in float32 with one rounding:
//
//     out[t, h * dv + d] = o[t, h, d] / sqrt(mean_d o[t, h, :]^2 + eps) * w[d] * silu(g[t, h * dv + d])      (gate_act 1: sigmoid(g))
#include "common.cuh"

template <typename T, typename TW>
__global__ void __launch_bounds__(128) gla_out_kernel(const float* __restrict__ o, const T* __restrict__ g, int g_stride,
                                                      const TW* __restrict__ w, T* __restrict__ out, int rows, int H, int dv,
                                                      float eps, int gate_act) {
    const int lane = threadIdx.x & 31;
    const int r = blockIdx.x * 4 + (threadIdx.x >> 5);       // (token, head)
    llb_grid_dependency_sync();
    if (r >= rows) return;
    const int t = r / H, h = r - t * H;
    const float* x = o + (size_t)r * dv;
    float ss = 0.f;
    for (int d = lane; d < dv; d += 32) ss += x[d] * x[d];
    ss = warp_sum(ss);
    const float inv = 1.0f / sqrtf(ss / (float)dv + eps);
    for (int d = lane; d < dv; d += 32) {
        float gv = to_f32(g[(size_t)t * g_stride + h * dv + d]);
        const float sg = 1.0f / (1.0f + expf(-gv));
        out[(size_t)r * dv + d] = from_f32<T>(x[d] * inv * to_f32(w[d]) * (gate_act == 1 ? sg : gv * sg));
    }
}

// bfloat16 gate and output, heads of up to 128 channels (a multiple of 4), rows of 8-byte pieces: a lane takes four neighbouring
// channels, a warp four (token, head) rows whose loads are in flight together.
constexpr int OUT_ROWS = 4;
template <typename TW>
__global__ void __launch_bounds__(128) gla_out_vec_kernel(const float* __restrict__ o, const bf16* __restrict__ g, int g_stride,
                                                          const TW* __restrict__ w, bf16* __restrict__ out, int rows, int H, int dv,
                                                          float eps, int gate_act) {
    const int lane = threadIdx.x & 31, d = lane * 4;
    const int r0 = (blockIdx.x * 4 + (threadIdx.x >> 5)) * OUT_ROWS;
    float wv[4] = {0.f, 0.f, 0.f, 0.f};
    if (d < dv)
#pragma unroll
        for (int e = 0; e < 4; ++e) wv[e] = to_f32(w[d + e]);
    llb_grid_dependency_sync();
    float4 x[OUT_ROWS];
    uint2 gate[OUT_ROWS];
#pragma unroll
    for (int k = 0; k < OUT_ROWS; ++k) {
        const int r = r0 + k, t = r / H;
        const bool in = r < rows && d < dv;
        x[k] = in ? *reinterpret_cast<const float4*>(o + (size_t)r * dv + d) : make_float4(0.f, 0.f, 0.f, 0.f);
        gate[k] = in ? *reinterpret_cast<const uint2*>(g + (size_t)t * g_stride + (r - t * H) * dv + d) : make_uint2(0u, 0u);
    }
#pragma unroll
    for (int k = 0; k < OUT_ROWS; ++k) {
        const float ss = warp_sum((x[k].x * x[k].x + x[k].y * x[k].y) + (x[k].z * x[k].z + x[k].w * x[k].w));
        if (r0 + k >= rows || d >= dv) continue;
        const float inv = 1.0f / sqrtf(ss / (float)dv + eps);
        const bf16* gv = reinterpret_cast<const bf16*>(&gate[k]);
        const float xv[4] = {x[k].x, x[k].y, x[k].z, x[k].w};
        uint2 y;
        bf16* yv = reinterpret_cast<bf16*>(&y);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const float gf = to_f32(gv[e]), sg = __fdividef(1.0f, 1.0f + __expf(-gf));      // (rounded to bfloat16 below)
            yv[e] = from_f32<bf16>(xv[e] * inv * wv[e] * (gate_act == 1 ? sg : gf * sg));
        }
        *reinterpret_cast<uint2*>(out + (size_t)(r0 + k) * dv + d) = y;
    }
}

LLB_API int llb_gla_out(const float* o, const void* g, int g_stride, const void* w, int w_dtype, void* out, int dtype,
                        int T, int H, int dv, float eps, int gate_act, cudaStream_t stream) {
    int rows = T * H;
    if (rows == 0) return 0;
    if (dtype == LLB_BF16 && dv % 4 == 0 && dv <= 128 && g_stride % 4 == 0 && !((uintptr_t)o & 15) && !(((uintptr_t)g | (uintptr_t)out) & 7)) {
        LLB_DISPATCH_DTYPE(w_dtype, TW, {
            llb_launch(gla_out_vec_kernel<TW>, dim3((rows + 4 * OUT_ROWS - 1) / (4 * OUT_ROWS)), dim3(128), 0, stream, o, (const bf16*)g,
                       g_stride, (const TW*)w, (bf16*)out, rows, H, dv, eps, gate_act);
        });
        return llb_status();
    }
    LLB_DISPATCH_DTYPE(dtype, TT, {
        LLB_DISPATCH_DTYPE(w_dtype, TW, {
            llb_launch(gla_out_kernel<TT, TW>, dim3((rows + 3) / 4), dim3(128), 0, stream, o, (const TT*)g, g_stride,
                       (const TW*)w, (TT*)out, rows, H, dv, eps, gate_act);
        });
    });
    return llb_status();
}
