// Grouped attention's row kernel: queries and keys rotated and narrowed, [key | value] rows put into the cache.
#include "qkv_rows.cuh"

namespace cq {

// One CTA per (row, section): the query heads, the key heads, the value heads.
template <typename A>
__global__ void __launch_bounds__(256) qkv_rows_kernel(const QkvRowsArgs a) {
    pdl_launch_dependents(); pdl_wait();
    qkv_section<A>(a, blockIdx.x, (a.pos_ptr ? *a.pos_ptr : a.pos0) + blockIdx.x, blockIdx.y, threadIdx.x, 256);
}
int launch_qkv_rows(int act, const QkvRowsArgs& a, int T, const LaunchCfg& cfg) {
    if (T < 1 || !qkv_rows_ok(a)) return (int)cudaErrorInvalidValue;
    const dim3 grid(T, 3);
    return act == ACT_F32 ? st_launch(qkv_rows_kernel<float>, grid, dim3(256), 0, cfg, a) : st_launch(qkv_rows_kernel<bf16>, grid, dim3(256), 0, cfg, a);
}

}  // namespace cq
