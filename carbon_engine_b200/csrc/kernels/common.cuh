// Shared declarations of the engine's CUDA kernels (sm_100a).
//
// Every launcher is an extern "C" function that takes raw device pointers and a stream, checks
// the sizes it is given, and returns 0 or a negative code after storing a message that
// ce_last_error() returns.  A launcher never allocates memory and never synchronises.
#pragma once
#include <cuda_runtime.h>
#include <cuda_bf16.h>
#include <stdint.h>

#define CE_OK 0
#define CE_ERR_SIZE -1      // a size this kernel refuses
#define CE_ERR_CUDA -2      // the launch itself failed
#define CE_ERR_ARG -3       // a null pointer or an unknown dtype

// dtype codes shared with the Python side
#define CE_F32 0
#define CE_BF16 1

#include <utility>

extern "C" const char* ce_last_error();
// Programmatic dependent launch: a kernel launched through ce_launch() may be scheduled while the
// kernel before it in the stream still runs.  Every kernel therefore begins with ce_pdl_begin():
// it lets its own dependents be scheduled early, and then waits until all grids before it are
// complete and their memory is visible, before it touches anything they wrote or still read.
// (Both instructions do nothing in a kernel launched the ordinary way.)
bool ce_pdl_enabled();
__device__ __forceinline__ void ce_pdl_launch_dependents() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void ce_pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void ce_pdl_begin() { ce_pdl_launch_dependents(); ce_pdl_wait(); }

template <typename... KArgs, typename... Args>
inline cudaError_t ce_launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream, Args&&... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = ce_pdl_enabled() ? 1 : 0;
    return cudaLaunchKernelEx(&cfg, kernel, std::forward<Args>(args)...);
}
int ce_fail(int code, const char* fmt, ...);
// Counts a launch under the kernel's name (ce_kernel_counts() lists them), so that a test or a
// measurement can see WHICH kernel took a shape.  Called by the launchers once per launch.
void ce_note(const char* kernel_name);
int ce_check_launch(const char* what);
int ce_sm_count();

// 2^x in one MUFU instruction (relative error about 2^-22; -inf gives 0).  exp2f() costs several
// instructions around the same MUFU; the bfloat16 attention kernels, whose probabilities are rounded to
// 8 bits of mantissa anyway, are bound by exactly those instructions.
// What a softmax row's sums are divided by, as its inverse.  M: the row's running maximum, L: its sum of 2^(s - M), both in
// the base-2 domain.  ``sinks`` (or null): a learned number per head whose exponential is one more term of the denominator,
// with no key and no value (given in the natural domain; it is neither scaled nor masked).  ``out_scale`` multiplies the result.
__device__ __forceinline__ float ce_softmax_inverse(float M, float L, const float* sinks, int h, float out_scale) {
    float shrink = 1.0f;
    if (sinks) {
        float sk = sinks[h] * 1.4426950408889634f, big = fmaxf(M, sk);
        shrink = M == -INFINITY ? 0.f : exp2f(M - big);
        L = L * shrink + exp2f(sk - big);
    }
    return (L > 0.f ? shrink / L : 0.f) * out_scale;
}

__device__ __forceinline__ float ce_exp2_fast(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// The clamped gated activation: g = min(gate, limit), u = up cut to [-limit, limit]; g sigmoid(alpha g) (u + 1).
__device__ __forceinline__ float ce_clamp_glu(float g, float u, float limit, float alpha) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.0f + expf(-alpha * g)) * (u + 1.0f);
}
// the same with the approximate exponential and reciprocal, for results that are rounded to bfloat16 right after
__device__ __forceinline__ float ce_clamp_glu_fast(float g, float u, float limit, float alpha) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return __fdividef(g, 1.0f + __expf(-alpha * g)) * (u + 1.0f);
}

// silu(gate) * up, exact and for results that are rounded to bfloat16 right after
__device__ __forceinline__ float ce_silu_glu(float g, float u) { return g / (1.0f + expf(-g)) * u; }
__device__ __forceinline__ float ce_silu_glu_fast(float g, float u) { return __fdividef(g, 1.0f + __expf(-g)) * u; }

template <typename T> struct CeType;
template <> struct CeType<float> {
    static __device__ __forceinline__ float load(const float* p) { return *p; }
    static __device__ __forceinline__ void store(float* p, float v) { *p = v; }
};
template <> struct CeType<__nv_bfloat16> {
    static __device__ __forceinline__ float load(const __nv_bfloat16* p) { return __bfloat162float(*p); }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
};

// four consecutive elements as float32
__device__ __forceinline__ float4 ce_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ce_load4(const __nv_bfloat16* p) {
    uint2 r = *reinterpret_cast<const uint2*>(p);
    float2 lo = __bfloat1622float2(*reinterpret_cast<__nv_bfloat162*>(&r.x)), hi = __bfloat1622float2(*reinterpret_cast<__nv_bfloat162*>(&r.y));
    return make_float4(lo.x, lo.y, hi.x, hi.y);
}

// Columns j .. j + 3 of a token's weighted sum of its experts' rows: sum_k weights[k] rows[pair_row[k]], in the order of k.
template <typename T>
__device__ __forceinline__ float4 ce_sum_picks4(const T* rows, int ld, const int* pair_row, const float* weights, int top, int j) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int k = 0; k < top; ++k) {
        const float w = weights[k];
        const float4 r = ce_load4(rows + (size_t)pair_row[k] * ld + j);
        v.x = fmaf(w, r.x, v.x); v.y = fmaf(w, r.y, v.y); v.z = fmaf(w, r.z, v.z); v.w = fmaf(w, r.w, v.w);
    }
    return v;
}

// Sum over a block in a fixed order: warp shuffles down, then warp 0 adds the warp sums in index
// order.  The result depends on blockDim only, never on the grid or on other rows.
__device__ __forceinline__ float ce_block_sum(float v, float* scratch /* >= 32 floats */) {
    for (int o = 16; o > 0; o >>= 1) v += __shfl_down_sync(0xffffffffu, v, o);
    int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = (blockDim.x + 31) >> 5;
    __syncthreads();
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    float total = 0.f;
    for (int w = 0; w < nwarp; ++w) total += scratch[w];
    return total;
}

__device__ __forceinline__ float ce_block_max(float v, float* scratch) {
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_down_sync(0xffffffffu, v, o));
    int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = (blockDim.x + 31) >> 5;
    __syncthreads();
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    float m = scratch[0];
    for (int w = 1; w < nwarp; ++w) m = fmaxf(m, scratch[w]);
    return m;
}
