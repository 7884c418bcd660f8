// Row-wise kernels of the layer-list designs: embedding rows, residual + norms, query / key-value latents, rotation.
#include "stack_dev.cuh"

namespace cq {

__device__ __forceinline__ void embed_row(const bf16* src, float* dst, int width) {
    for (int i = threadIdx.x; i < width; i += blockDim.x) dst[i] = __bfloat162float(src[i]);
}
__global__ void __launch_bounds__(256) st_embed_kernel(const bf16* __restrict__ table, int pitch, const int* __restrict__ tokens, float* __restrict__ x, int ldx, int width) {
    pdl_launch_dependents(); pdl_wait();
    embed_row(table + (size_t)tokens[blockIdx.x] * pitch, x + (size_t)blockIdx.x * ldx, width);
}
int launch_st_embed(const bf16* table, int pitch, const int* tokens, float* x, int ldx, int width, int T, const LaunchCfg& cfg) {
    return st_launch(st_embed_kernel, dim3(T), dim3(256), 0, cfg, table, pitch, tokens, x, ldx, width);
}

// One CTA: thread 0 takes over what the host left in the mailbox before any dependent launch is released (as
// embed_step_kernel does for the models of the table).
__global__ void __launch_bounds__(256) st_embed_step_kernel(const bf16* __restrict__ table, int pitch, StepCtl* ctl, float* __restrict__ x, int width) {
    if (threadIdx.x == 0 && ctl->hio && !ctl->auto_advance) {
        int sq, tk, ps, hl;
        asm volatile("ld.volatile.global.v4.s32 {%0,%1,%2,%3}, [%4];" : "=r"(sq), "=r"(tk), "=r"(ps), "=r"(hl) : "l"(ctl->hio) : "memory");
        if (sq != ctl->io_seq) { ctl->token = tk; ctl->pos = ps; ctl->hist_len = hl; ctl->io_seq = sq; }
        __threadfence();
    }
    __syncthreads();
    pdl_launch_dependents();
    embed_row(table + (size_t)(*(volatile int*)&ctl->token) * pitch, x, width);
}
int launch_st_embed_step(const bf16* table, int pitch, StepCtl* ctl, float* x, int width, const LaunchCfg& cfg) {
    return st_launch(st_embed_step_kernel, dim3(1), dim3(256), 0, cfg, table, pitch, ctl, x, width);
}

// ---- x += rmsnorm(y), then one or two norms of x ------------------------------------------------------------------------
// One CTA per row; a thread keeps its elements (one in 256) in registers up to a width of 8192 and re-reads them beyond.
template <typename A>
__global__ void __launch_bounds__(256) st_norms_kernel(const NormRowsArgs a) {
    __shared__ float red[40];
    pdl_launch_dependents(); pdl_wait();
    const int t = blockIdx.x;
    float* x = a.x + (size_t)(a.rows ? a.rows[t] : t) * a.ldx;
    if (a.y) {
        const float* y = a.y + (size_t)t * a.ldy;
        float ss = 0.f;
        for (int i = threadIdx.x; i < a.width; i += 256) ss += y[i] * y[i];
        const float inv = inv_rms(cta_sum(ss, red), a.width, a.eps);
        for (int i = threadIdx.x; i < a.width; i += 256) x[i] += y[i] * inv * a.y_w[i];      // the same thread reads it below
    }
    if (a.n_out == 0) return;
    float ss = 0.f;
    for (int i = threadIdx.x; i < a.width; i += 256) ss += x[i] * x[i];
    const float inv = inv_rms(cta_sum(ss, red), a.width, a.eps);
    for (int k = 0; k < a.n_out; ++k) {
        A* o = reinterpret_cast<A*>(a.out[k]) + (size_t)t * a.ldo;
        for (int i = threadIdx.x; i < a.ldo; i += 256) o[i] = to_act<A>(i < a.width ? x[i] * inv * a.w[k][i] : 0.f);
    }
}
int launch_st_norms(int act, const NormRowsArgs& a, int T, const LaunchCfg& cfg) {
    return act == ACT_F32 ? st_launch(st_norms_kernel<float>, dim3(T), dim3(256), 0, cfg, a) : st_launch(st_norms_kernel<bf16>, dim3(T), dim3(256), 0, cfg, a);
}

template <typename A>
__global__ void __launch_bounds__(256) st_narrow_kernel(const float* __restrict__ x, int ldx, A* __restrict__ out, int ldo) {
    pdl_launch_dependents(); pdl_wait();
    for (int i = threadIdx.x; i < ldo; i += 256) out[(size_t)blockIdx.x * ldo + i] = to_act<A>(i < ldx ? x[(size_t)blockIdx.x * ldx + i] : 0.f);
}
int launch_st_narrow(int act, const float* x, int ldx, void* out, int ldo, int T, const LaunchCfg& cfg) {
    return act == ACT_F32 ? st_launch(st_narrow_kernel<float>, dim3(T), dim3(256), 0, cfg, x, ldx, (float*)out, ldo) : st_launch(st_narrow_kernel<bf16>, dim3(T), dim3(256), 0, cfg, x, ldx, (bf16*)out, ldo);
}

// ---- query latent and cache row ---------------------------------------------------------------------------------------
template <typename A>
__global__ void __launch_bounds__(256) st_latent_rows_kernel(const LatentRowsArgs a) {
    __shared__ float red[40];
    pdl_launch_dependents(); pdl_wait();
    const int t = blockIdx.x;
    if (blockIdx.y == 0) {
        const float* q = a.dq + (size_t)t * a.ld;
        float ss = 0.f;
        for (int i = threadIdx.x; i < a.q_rank; i += 256) ss += q[i] * q[i];
        const float inv = inv_rms(cta_sum(ss, red), a.q_rank, a.eps);
        A* o = reinterpret_cast<A*>(a.cq) + (size_t)t * a.ldcq;
        for (int i = threadIdx.x; i < a.ldcq; i += 256) o[i] = to_act<A>(i < a.q_rank ? q[i] * inv * a.dq_w[i] : 0.f);
    } else {
        const int pos = (a.pos_ptr ? *a.pos_ptr : a.pos0) + t;
        const float* kv = a.dkv + (size_t)t * a.ld;
        float ss = 0.f;
        for (int i = threadIdx.x; i < a.kv_rank; i += 256) ss += kv[i] * kv[i];
        const float inv = inv_rms(cta_sum(ss, red), a.kv_rank, a.eps);
        A* o = reinterpret_cast<A*>(a.cache) + (size_t)pos * a.ldc;
        for (int i = threadIdx.x; i < a.kv_rank; i += 256) o[i] = to_act<A>(kv[i] * inv * a.dkv_w[i]);
        const int half = a.rot_dim / 2;
        for (int i = threadIdx.x; i < half; i += 256) {
            const float2 cs = a.rot[(size_t)pos * half + i];
            const float u = kv[a.kr_off + i], v = kv[a.kr_off + half + i];
            o[a.kr_off + i] = to_act<A>(u * cs.x - v * cs.y);
            o[a.kr_off + half + i] = to_act<A>(v * cs.x + u * cs.y);
        }
    }
}
int launch_st_latent_rows(int act, const LatentRowsArgs& a, int T, const LaunchCfg& cfg) {
    const dim3 grid(T, a.dkv ? 2 : 1);
    return act == ACT_F32 ? st_launch(st_latent_rows_kernel<float>, grid, dim3(256), 0, cfg, a) : st_launch(st_latent_rows_kernel<bf16>, grid, dim3(256), 0, cfg, a);
}

// ---- rotation of the query heads --------------------------------------------------------------------------------------
template <typename A>
__global__ void __launch_bounds__(256) st_rope_q_kernel(const RopeQArgs a) {
    pdl_launch_dependents(); pdl_wait();
    const int t = blockIdx.x, half = a.rot_dim / 2;
    const int pos = (a.pos_ptr ? *a.pos_ptr : a.pos0) + t;
    const float* in = a.in + (size_t)t * a.ld;
    A* out = reinterpret_cast<A*>(a.out) + (size_t)t * a.ld;
    for (int i = threadIdx.x; i < a.heads * a.head_pitch; i += 256) {
        const int c = i % a.head_pitch, r = c - a.rot_off;
        if (r < 0 || r >= a.rot_dim) out[i] = to_act<A>(in[i]);
        else if (r < half) {
            const float2 cs = a.rot[(size_t)pos * half + r];
            const float u = in[i], v = in[i + half];
            out[i] = to_act<A>(u * cs.x - v * cs.y);
            out[i + half] = to_act<A>(v * cs.x + u * cs.y);
        }
    }
}
int launch_st_rope_q(int act, const RopeQArgs& a, int T, const LaunchCfg& cfg) {
    return act == ACT_F32 ? st_launch(st_rope_q_kernel<float>, dim3(T), dim3(256), 0, cfg, a) : st_launch(st_rope_q_kernel<bf16>, dim3(T), dim3(256), 0, cfg, a);
}

// ---- rotation table -----------------------------------------------------------------------------------------------------
// Frequency and angle in double, so that a far position's angle carries no more than the rounding of its cosine and sine.
__global__ void rot_table_kernel(float2* table, int n_pos, int dims, double base) {
    const int half = dims / 2;
    const size_t n = (size_t)n_pos * half;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
        const double a = (double)(i / half) * pow(base, -2.0 * (double)(i % half) / (double)dims);
        double s, c;
        sincos(a, &s, &c);
        table[i] = make_float2((float)c, (float)s);
    }
}
int launch_rot_table(float2* table, int n_pos, int dims, double base, const LaunchCfg& cfg) {
    return st_launch(rot_table_kernel, dim3(1024), dim3(128), 0, cfg, table, n_pos, dims, base);
}

}  // namespace cq
