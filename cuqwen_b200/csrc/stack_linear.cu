// Matrix products of the layer-list designs on the CUDA cores, any sizes, both activation types, float32 accumulation:
// the 32-bit mode's only path.  (bfloat16 prefill uses prefill_gemm.cu, bfloat16 decode gemv_bf16.cu.)
#include "stack_dev.cuh"

namespace cq {

template <typename A>
__device__ __forceinline__ void lin_store(const LinArgs& a, int t, int r, float v) {
    const size_t o = (size_t)t * a.ldo + r;
    switch (a.epi) {
        case LIN_F32: reinterpret_cast<float*>(a.out)[o] = v; break;
        case LIN_ACT: reinterpret_cast<A*>(a.out)[o] = to_act<A>(v); break;
        case LIN_RELU2: { const float p = fmaxf(v, 0.f); reinterpret_cast<A*>(a.out)[o] = to_act<A>(p * p); break; }
        case LIN_ADD: reinterpret_cast<float*>(a.out)[o] += a.c0 * v; break;
        case LIN_DECAY: reinterpret_cast<float*>(a.out)[o] = expf(-expf(v + a.bias[r])); break;
        case LIN_CAP: reinterpret_cast<float*>(a.out)[o] = a.c0 * tanhf(v / a.c0); break;
        case LIN_GELU_SIDE: {
            const float e = r < a.side_dim ? __bfloat162float(a.side[(size_t)a.tokens[t] * a.side_pitch + r]) : 0.f;
            reinterpret_cast<A*>(a.out)[o] = to_act<A>(gelu_tanh_f(v) * e);
            break;
        }
    }
}

// One token: a warp per output row.
template <typename A>
__global__ void __launch_bounds__(256) st_gemv_kernel(const LinArgs a) {
    pdl_launch_dependents(); pdl_wait();
    const int r = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (r >= a.R) return;
    float s = 0.f;
    for (int part = 0; part < (a.w2 ? 2 : 1); ++part) {
        const A* x = reinterpret_cast<const A*>(part ? a.x2 : a.x);
        const bf16* w = part ? a.w2 + (size_t)r * a.pitch2 : a.w + (size_t)r * a.pitch;
        const int K = part ? a.K2 : a.K;
        for (int k = lane; k < K; k += 32) s = fmaf(act_f(x[k]), __bfloat162float(w[k]), s);
    }
    s = warp_sum(s);
    if (lane == 0) lin_store<A>(a, 0, r, s);
}

// Many tokens: 64 x 64 tiles, 16 columns of K at a time, a 4 x 4 block of the tile per thread.
template <typename A>
__global__ void __launch_bounds__(256) st_gemm_kernel(const LinArgs a) {
    __shared__ float xs[16][65], ws[16][65];
    pdl_launch_dependents(); pdl_wait();
    const int t0 = blockIdx.y * 64, r0 = blockIdx.x * 64, tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {};
    for (int part = 0; part < (a.w2 ? 2 : 1); ++part) {
        const A* x = reinterpret_cast<const A*>(part ? a.x2 : a.x);
        const bf16* w = part ? a.w2 : a.w;
        const int K = part ? a.K2 : a.K, ldx = part ? a.ldx2 : a.ldx, pitch = part ? a.pitch2 : a.pitch;
        for (int k0 = 0; k0 < K; k0 += 16) {
            for (int i = threadIdx.x; i < 1024; i += 256) {
                const int row = i >> 4, k = i & 15;
                xs[k][row] = t0 + row < a.T && k0 + k < K ? act_f(x[(size_t)(t0 + row) * ldx + k0 + k]) : 0.f;
                ws[k][row] = r0 + row < a.R && k0 + k < K ? __bfloat162float(w[(size_t)(r0 + row) * pitch + k0 + k]) : 0.f;
            }
            __syncthreads();
#pragma unroll
            for (int k = 0; k < 16; ++k) {
                float xv[4], wv[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) { xv[i] = xs[k][ty * 4 + i]; wv[i] = ws[k][tx + 16 * i]; }
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xv[i], wv[j], acc[i][j]);
            }
            __syncthreads();
        }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int t = t0 + ty * 4 + i, r = r0 + tx + 16 * j;
            if (t < a.T && r < a.R) lin_store<A>(a, t, r, acc[i][j]);
        }
}

int launch_st_linear(int act, const LinArgs& a, const LaunchCfg& cfg) {
    if (a.T < 1 || a.R < 1 || a.K < 1 || !a.x || !a.w || !a.out || a.epi == LIN_GLU) return (int)cudaErrorInvalidValue;
    if (a.T == 1) {
        const dim3 grid((a.R + 7) / 8);
        return act == ACT_F32 ? st_launch(st_gemv_kernel<float>, grid, dim3(256), 0, cfg, a) : st_launch(st_gemv_kernel<bf16>, grid, dim3(256), 0, cfg, a);
    }
    const dim3 grid((a.R + 63) / 64, (a.T + 63) / 64);
    return act == ACT_F32 ? st_launch(st_gemm_kernel<float>, grid, dim3(256), 0, cfg, a) : st_launch(st_gemm_kernel<bf16>, grid, dim3(256), 0, cfg, a);
}

}  // namespace cq
