// Row-wise kernels of the layer-list designs: embedding rows, residual + norms, query / key-value latents, rotation.
#include "stack_dev.cuh"

namespace cq {

__device__ __forceinline__ void embed_row(const bf16* src, float* dst, int width, float scale) {
    for (int i = threadIdx.x; i < (width + 7) / 8; i += blockDim.x) {      // rows are padded with zeros to a multiple of eight
        float v[8];
        unpack8(ldg_stream(src + 8 * i), v);
#pragma unroll
        for (int k = 0; k < 8; ++k) v[k] *= scale;
        store4(dst + 8 * i, make_float4(v[0], v[1], v[2], v[3]));
        store4(dst + 8 * i + 4, make_float4(v[4], v[5], v[6], v[7]));
    }
}
__global__ void __launch_bounds__(256) st_embed_kernel(const bf16* __restrict__ table, int pitch, const int* __restrict__ tokens, float* __restrict__ x, int ldx, int width, float scale) {
    pdl_launch_dependents(); pdl_wait();
    embed_row(table + (size_t)tokens[blockIdx.x] * pitch, x + (size_t)blockIdx.x * ldx, width, scale);
}
int launch_st_embed(const bf16* table, int pitch, const int* tokens, float* x, int ldx, int width, float scale, int T, const LaunchCfg& cfg) {
    return st_launch(st_embed_kernel, dim3(T), dim3(256), 0, cfg, table, pitch, tokens, x, ldx, width, scale);
}

// One CTA: thread 0 takes over what the host left in the mailbox before any dependent launch is released (as
// embed_step_kernel does for the models of the table).
__global__ void __launch_bounds__(256) st_embed_step_kernel(const bf16* __restrict__ table, int pitch, StepCtl* ctl, float* __restrict__ x, int width, float scale) {
    if (threadIdx.x == 0 && ctl->hio && !ctl->auto_advance) {
        int sq, tk, ps, hl;
        asm volatile("ld.volatile.global.v4.s32 {%0,%1,%2,%3}, [%4];" : "=r"(sq), "=r"(tk), "=r"(ps), "=r"(hl) : "l"(ctl->hio) : "memory");
        if (sq != ctl->io_seq) { ctl->token = tk; ctl->pos = ps; ctl->hist_len = hl; ctl->io_seq = sq; }
        __threadfence();
    }
    __syncthreads();
    pdl_launch_dependents();
    embed_row(table + (size_t)(*(volatile int*)&ctl->token) * pitch, x, width, scale);
}
int launch_st_embed_step(const bf16* table, int pitch, StepCtl* ctl, float* x, int width, float scale, const LaunchCfg& cfg) {
    return st_launch(st_embed_step_kernel, dim3(1), dim3(256), 0, cfg, table, pitch, ctl, x, width, scale);
}

// ---- x += rmsnorm(y), then one or two norms of x ------------------------------------------------------------------------
// One CTA per row, the row in registers: a thread owns the float4 units tid, tid + 256, ... (NV of them at the most; rows are
// padded with zeros to a multiple of eight).  NV = 0: any width, the row re-read from memory instead.
template <typename A, int NV>
__global__ void __launch_bounds__(256) st_norms_kernel(const NormRowsArgs a) {
    __shared__ float red[40];
    pdl_launch_dependents(); pdl_wait();
    const int t = blockIdx.x, tid = threadIdx.x, n4 = (a.width + 3) / 4, o4 = a.ldo / 4;
    float4* x = reinterpret_cast<float4*>(a.x + (size_t)(a.rows ? a.rows[t] : t) * a.ldx);
    const float4* y = a.y ? reinterpret_cast<const float4*>(a.y + (size_t)t * a.ldy) : nullptr;
    constexpr int N = NV > 0 ? NV : 1;
    float4 v[N];
    float ss = 0.f;
    if (NV > 0) {
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] = i * 256 + tid < n4 ? x[i * 256 + tid] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    if (y) {
        const float4* yw = reinterpret_cast<const float4*>(a.y_w);
        auto add = [&](float4 p, float4 u, float inv, float4 w) { return make_float4(p.x + u.x * inv * w.x, p.y + u.y * inv * w.y, p.z + u.z * inv * w.z, p.w + u.w * inv * w.w); };
        float sy = 0.f;
        if (NV > 0) {
            float4 u[N];
#pragma unroll
            for (int i = 0; i < N; ++i) { u[i] = i * 256 + tid < n4 ? y[i * 256 + tid] : make_float4(0.f, 0.f, 0.f, 0.f); sy += dot4(u[i], u[i]); }
            const float inv = inv_rms(cta_sum(sy, red), a.width, a.eps);
#pragma unroll
            for (int i = 0; i < N; ++i) if (i * 256 + tid < n4) { v[i] = add(v[i], u[i], inv, yw[i * 256 + tid]); x[i * 256 + tid] = v[i]; }
        } else {
            for (int i = tid; i < n4; i += 256) sy += dot4(y[i], y[i]);
            const float inv = inv_rms(cta_sum(sy, red), a.width, a.eps);
            for (int i = tid; i < n4; i += 256) x[i] = add(x[i], y[i], inv, yw[i]);          // the same thread reads it below
        }
    }
    if (a.n_out == 0) return;
    if (NV > 0) {
#pragma unroll
        for (int i = 0; i < N; ++i) ss += dot4(v[i], v[i]);
    } else for (int i = tid; i < n4; i += 256) ss += dot4(x[i], x[i]);
    const float inv = inv_rms(cta_sum(ss, red), a.width, a.eps);
    for (int k = 0; k < a.n_out; ++k) {
        A* o = reinterpret_cast<A*>(a.out[k]) + (size_t)t * a.ldo;
        const float4* w = reinterpret_cast<const float4*>(a.w[k]);
        auto put = [&](int i, float4 p) {
            if (i < n4) { const float4 g = w[i]; p = make_float4(p.x * inv * g.x, p.y * inv * g.y, p.z * inv * g.z, p.w * inv * g.w); }
            if (i < o4) store4(o + 4 * i, p);
        };
        if (NV > 0) {
#pragma unroll
            for (int i = 0; i < N; ++i) put(i * 256 + tid, v[i]);
        } else for (int i = tid; i < o4; i += 256) put(i, i < n4 ? x[i] : make_float4(0.f, 0.f, 0.f, 0.f));
    }
}
template <typename A>
static int go_norms(const NormRowsArgs& a, int T, const LaunchCfg& cfg) {
    const int nv = (a.ldo > a.width ? a.ldo : a.width) / 4;
    if (nv <= 2 * 256) return st_launch(st_norms_kernel<A, 2>, dim3(T), dim3(256), 0, cfg, a);
    if (nv <= 4 * 256) return st_launch(st_norms_kernel<A, 4>, dim3(T), dim3(256), 0, cfg, a);
    if (nv <= 8 * 256) return st_launch(st_norms_kernel<A, 8>, dim3(T), dim3(256), 0, cfg, a);
    return st_launch(st_norms_kernel<A, 0>, dim3(T), dim3(256), 0, cfg, a);
}
int launch_st_norms(int act, const NormRowsArgs& a, int T, const LaunchCfg& cfg) { return act == ACT_F32 ? go_norms<float>(a, T, cfg) : go_norms<bf16>(a, T, cfg); }

template <typename A>
__global__ void __launch_bounds__(256) st_narrow_kernel(const float* __restrict__ x, int ldx, A* __restrict__ out, int ldo) {
    pdl_launch_dependents(); pdl_wait();
    for (int i = threadIdx.x; i < ldo; i += 256) out[(size_t)blockIdx.x * ldo + i] = to_act<A>(i < ldx ? x[(size_t)blockIdx.x * ldx + i] : 0.f);
}
int launch_st_narrow(int act, const float* x, int ldx, void* out, int ldo, int T, const LaunchCfg& cfg) {
    return act == ACT_F32 ? st_launch(st_narrow_kernel<float>, dim3(T), dim3(256), 0, cfg, x, ldx, (float*)out, ldo) : st_launch(st_narrow_kernel<bf16>, dim3(T), dim3(256), 0, cfg, x, ldx, (bf16*)out, ldo);
}

// ---- query latent and cache row ---------------------------------------------------------------------------------------
// One CTA of 128 threads per (row, half): blockIdx.y 0 the query latent, 1 the cache row.  A row of up to 2048 values stays in
// registers (four float4 units a thread), a longer one is re-read.
template <typename A>
__global__ void __launch_bounds__(128) st_latent_rows_kernel(const LatentRowsArgs a) {
    __shared__ float red[40];
    pdl_launch_dependents(); pdl_wait();
    const int t = blockIdx.x, tid = threadIdx.x;
    const bool kv = a.dq == nullptr || blockIdx.y == 1;
    const int n = kv ? a.kv_rank : a.q_rank, n4 = (n + 3) / 4;
    const float* src = (kv ? a.dkv : a.dq) + (size_t)t * a.ld;
    const float4 *s4 = reinterpret_cast<const float4*>(src), *w4 = reinterpret_cast<const float4*>(kv ? a.dkv_w : a.dq_w);
    const int pos = (a.pos_ptr ? *a.pos_ptr : a.pos0) + t;
    A* o = kv ? reinterpret_cast<A*>(a.cache) + (size_t)pos * a.ldc : reinterpret_cast<A*>(a.cq) + (size_t)t * a.ldcq;
    float4 v[4];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) { v[i] = i * 128 + tid < n4 ? s4[i * 128 + tid] : make_float4(0.f, 0.f, 0.f, 0.f); ss += dot4(v[i], v[i]); }
    for (int i = 512 + tid; i < n4; i += 128) ss += dot4(s4[i], s4[i]);
    const float inv = inv_rms(cta_sum(ss, red), n, a.eps);
    auto put = [&](int i, float4 p) { const float4 g = w4[i]; store4(o + 4 * i, make_float4(p.x * inv * g.x, p.y * inv * g.y, p.z * inv * g.z, p.w * inv * g.w)); };
#pragma unroll
    for (int i = 0; i < 4; ++i) if (i * 128 + tid < n4) put(i * 128 + tid, v[i]);
    for (int i = 512 + tid; i < n4; i += 128) put(i, s4[i]);
    if (!kv) return;
    const int half = a.rot_dim / 2;
    for (int i = tid; i < half; i += 128) {
        const float2 cs = a.rot[(size_t)pos * half + i];
        const float p = src[a.kr_off + i], q = src[a.kr_off + half + i];
        o[a.kr_off + i] = to_act<A>(p * cs.x - q * cs.y);
        o[a.kr_off + half + i] = to_act<A>(q * cs.x + p * cs.y);
    }
}
int launch_st_latent_rows(int act, const LatentRowsArgs& a, int T, const LaunchCfg& cfg) {
    const dim3 grid(T, a.dkv && a.dq ? 2 : 1);
    return act == ACT_F32 ? st_launch(st_latent_rows_kernel<float>, grid, dim3(128), 0, cfg, a) : st_launch(st_latent_rows_kernel<bf16>, grid, dim3(128), 0, cfg, a);
}

// ---- rotation of the query heads --------------------------------------------------------------------------------------
template <typename A>
__global__ void __launch_bounds__(256) st_rope_q_kernel(const RopeQArgs a) {
    pdl_launch_dependents(); pdl_wait();
    const int t = blockIdx.x, half = a.rot_dim / 2;
    const int pos = (a.pos_ptr ? *a.pos_ptr : a.pos0) + t;
    const float* in = a.in + (size_t)t * a.ld;
    A* out = reinterpret_cast<A*>(a.out) + (size_t)t * a.ld;
    // rot_off and head_pitch are multiples of eight; the padding behind the rotated part is never read
    const int units = a.rot_off / 4;
    for (int i = threadIdx.x; i < a.heads * units; i += 256) {
        const int o = i / units * a.head_pitch + i % units * 4;
        store4(out + o, *reinterpret_cast<const float4*>(in + o));
    }
    for (int i = threadIdx.x; i < a.heads * half; i += 256) {
        const int r = i % half, o = i / half * a.head_pitch + a.rot_off + r;
        const float2 cs = a.rot[(size_t)pos * half + r];
        const float u = in[o], v = in[o + half];
        out[o] = to_act<A>(u * cs.x - v * cs.y);
        out[o + half] = to_act<A>(v * cs.x + u * cs.y);
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
