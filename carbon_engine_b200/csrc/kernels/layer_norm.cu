// Layer norm with weight and bias, RMS norms that add into the residual stream, the RMS norm of a weighted residual plus a
// sublayer's output, the tanh cap of a row of numbers, a copy of a run of float32 columns into the activation dtype, and the gate of a per-token side input.
//
// All arithmetic is float32; a result is rounded once, at the store.  Sums over a row are taken by one block in
// an order that depends on the row's width only.
#include "common.cuh"

// ---------------------------------------------------------------------------------------------
// y = (x - mean) / sqrt(var + eps) * w + b, var the mean of the squared deviations (two passes over the row,
// which is kept in registers when it fits).  rows: optional gather of the rows to normalise.
// ---------------------------------------------------------------------------------------------
#define LN_MAX_PER_THREAD 16

template <typename T>
__global__ void layernorm_kernel(const float* __restrict__ x, const float* __restrict__ w, const float* __restrict__ b,
                                 T* __restrict__ out, const int* __restrict__ rows, int H, float eps) {
    ce_pdl_begin();
    __shared__ float scratch[32];
    int r = blockIdx.x;
    const float* xr = x + (size_t)(rows ? rows[r] : r) * H;
    float v[LN_MAX_PER_THREAD];
    float s = 0.f;
    int n = 0;
    for (int j = threadIdx.x; j < H; j += blockDim.x, ++n) {
        float e = xr[j];
        if (n < LN_MAX_PER_THREAD) v[n] = e;
        s += e;
    }
    float mean = ce_block_sum(s, scratch) / (float)H;
    float q = 0.f;
    n = 0;
    for (int j = threadIdx.x; j < H; j += blockDim.x, ++n) {
        float e = (n < LN_MAX_PER_THREAD ? v[n] : xr[j]) - mean;
        q = fmaf(e, e, q);
    }
    float inv = 1.0f / sqrtf(ce_block_sum(q, scratch) / (float)H + eps);
    n = 0;
    for (int j = threadIdx.x; j < H; j += blockDim.x, ++n) {
        float e = (n < LN_MAX_PER_THREAD ? v[n] : xr[j]) - mean;
        CeType<T>::store(out + (size_t)r * H + j, e * inv * w[j] + b[j]);
    }
}

// The same with float4 loads for widths in multiples of 4 up to 4 * 1024 * LNV_MAX: a thread keeps its float4s in registers.
#define LNV_MAX 4
template <typename T>
__global__ void layernorm_vec_kernel(const float* __restrict__ x, const float* __restrict__ w, const float* __restrict__ b,
                                     T* __restrict__ out, const int* __restrict__ rows, int H, float eps) {
    ce_pdl_begin();
    __shared__ float scratch[32];
    int r = blockIdx.x, H4 = H >> 2;
    const float4* xr = reinterpret_cast<const float4*>(x + (size_t)(rows ? rows[r] : r) * H);
    float4 v[LNV_MAX];
    float s = 0.f;
#pragma unroll
    for (int n = 0; n < LNV_MAX; ++n) {
        int j = threadIdx.x + n * blockDim.x;
        v[n] = j < H4 ? xr[j] : make_float4(0.f, 0.f, 0.f, 0.f);
        s += (v[n].x + v[n].y) + (v[n].z + v[n].w);
    }
    float mean = ce_block_sum(s, scratch) / (float)H;
    float q = 0.f;
#pragma unroll
    for (int n = 0; n < LNV_MAX; ++n) {
        int j = threadIdx.x + n * blockDim.x;
        if (j < H4) {
            v[n].x -= mean; v[n].y -= mean; v[n].z -= mean; v[n].w -= mean;
            q += (v[n].x * v[n].x + v[n].y * v[n].y) + (v[n].z * v[n].z + v[n].w * v[n].w);
        }
    }
    float inv = 1.0f / sqrtf(ce_block_sum(q, scratch) / (float)H + eps);
    const float4* w4 = reinterpret_cast<const float4*>(w);
    const float4* b4 = reinterpret_cast<const float4*>(b);
#pragma unroll
    for (int n = 0; n < LNV_MAX; ++n) {
        int j = threadIdx.x + n * blockDim.x;
        if (j < H4) {
            float4 ww = w4[j], bb = b4[j];
            T* o = out + (size_t)r * H + 4 * j;
            CeType<T>::store(o, v[n].x * inv * ww.x + bb.x); CeType<T>::store(o + 1, v[n].y * inv * ww.y + bb.y);
            CeType<T>::store(o + 2, v[n].z * inv * ww.z + bb.z); CeType<T>::store(o + 3, v[n].w * inv * ww.w + bb.w);
        }
    }
}

extern "C" int ce_layernorm(const float* x, const float* w, const float* b, void* out, int out_dtype, const int* rows,
                            int R, int H, float eps, cudaStream_t stream) {
    if (R == 0) return CE_OK;
    if (!x || !w || !b || !out) return ce_fail(CE_ERR_ARG, "ce_layernorm: null pointer");
    if (H <= 0) return ce_fail(CE_ERR_SIZE, "ce_layernorm: width %d", H);
    if (out_dtype != CE_F32 && out_dtype != CE_BF16) return ce_fail(CE_ERR_ARG, "ce_layernorm: unknown dtype %d", out_dtype);
    if (H % 4 == 0 && H >= 256 && ((((uintptr_t)x | (uintptr_t)w | (uintptr_t)b) & 15) == 0)) {
        int H4 = H / 4, vt = H4 >= 2048 ? 1024 : H4 >= 512 ? 512 : H4 >= 256 ? 256 : 128;
        if (H4 <= vt * LNV_MAX) {
            ce_note("layernorm_vec_kernel");
            if (out_dtype == CE_F32) ce_launch(layernorm_vec_kernel<float>, R, vt, 0, stream, x, w, b, (float*)out, rows, H, eps);
            else ce_launch(layernorm_vec_kernel<__nv_bfloat16>, R, vt, 0, stream, x, w, b, (__nv_bfloat16*)out, rows, H, eps);
            return ce_check_launch("ce_layernorm");
        }
    }
    int threads = H >= 4096 ? 512 : H >= 1024 ? 256 : 128;
    ce_note("layernorm_kernel");
    if (out_dtype == CE_F32) ce_launch(layernorm_kernel<float>, R, threads, 0, stream, x, w, b, (float*)out, rows, H, eps);
    else if (out_dtype == CE_BF16) ce_launch(layernorm_kernel<__nv_bfloat16>, R, threads, 0, stream, x, w, b, (__nv_bfloat16*)out, rows, H, eps);
    else return ce_fail(CE_ERR_ARG, "ce_layernorm: unknown dtype %d", out_dtype);
    return ce_check_launch("ce_layernorm");
}

// ---------------------------------------------------------------------------------------------
// x[t] += y[t] / sqrt(mean(y[t]^2) + eps) * w      (y float32, x the float32 residual stream)
// ---------------------------------------------------------------------------------------------
__global__ void rmsnorm_add_kernel(const float* __restrict__ y, const float* __restrict__ w, float* __restrict__ x,
                                   __nv_bfloat16* __restrict__ xb, int H, float eps) {
    ce_pdl_begin();
    __shared__ float scratch[32];
    int t = blockIdx.x;
    const float* yr = y + (size_t)t * H;
    float q = 0.f;
    for (int j = threadIdx.x; j < H; j += blockDim.x) q = fmaf(yr[j], yr[j], q);
    float inv = 1.0f / sqrtf(ce_block_sum(q, scratch) / (float)H + eps);
    for (int j = threadIdx.x; j < H; j += blockDim.x) {
        float v = x[(size_t)t * H + j] + yr[j] * inv * w[j];
        x[(size_t)t * H + j] = v;
        if (xb) xb[(size_t)t * H + j] = __float2bfloat16_rn(v);
    }
}

// The same with float4 loads, y kept in registers between the two passes (widths in multiples of 4 up to 4 * threads * LNV_MAX)
__global__ void rmsnorm_add_vec_kernel(const float* __restrict__ y, const float* __restrict__ w, float* __restrict__ x,
                                       __nv_bfloat16* __restrict__ xb, int H, float eps) {
    ce_pdl_begin();
    __shared__ float scratch[32];
    int t = blockIdx.x, H4 = H >> 2;
    const float4* yr = reinterpret_cast<const float4*>(y + (size_t)t * H);
    float4 v[LNV_MAX];
    float q = 0.f;
#pragma unroll
    for (int n = 0; n < LNV_MAX; ++n) {
        int j = threadIdx.x + n * blockDim.x;
        v[n] = j < H4 ? yr[j] : make_float4(0.f, 0.f, 0.f, 0.f);
        q += (v[n].x * v[n].x + v[n].y * v[n].y) + (v[n].z * v[n].z + v[n].w * v[n].w);
    }
    float inv = 1.0f / sqrtf(ce_block_sum(q, scratch) / (float)H + eps);
    float4* xr = reinterpret_cast<float4*>(x + (size_t)t * H);
    const float4* w4 = reinterpret_cast<const float4*>(w);
#pragma unroll
    for (int n = 0; n < LNV_MAX; ++n) {
        int j = threadIdx.x + n * blockDim.x;
        if (j < H4) {
            float4 xv = xr[j], ww = w4[j];
            xv.x += v[n].x * inv * ww.x; xv.y += v[n].y * inv * ww.y; xv.z += v[n].z * inv * ww.z; xv.w += v[n].w * inv * ww.w;
            xr[j] = xv;
            if (xb) {
                __nv_bfloat162 lo = __floats2bfloat162_rn(xv.x, xv.y), hi = __floats2bfloat162_rn(xv.z, xv.w);
                uint2 packed = make_uint2(*reinterpret_cast<unsigned*>(&lo), *reinterpret_cast<unsigned*>(&hi));
                reinterpret_cast<uint2*>(xb + (size_t)t * H)[j] = packed;
            }
        }
    }
}

// The same, and the NEXT norm of the new x in the same pass:  y may still owe a bias (float32 [H] or null);
//   x[t] += (y[t] + bias) / sqrt(mean((y[t] + bias)^2) + eps) * w;     h[t] = x[t] / sqrt(mean(x[t]^2) + eps2) * w2
// h (or null: no next norm) is float32 or bfloat16.  VEC: float4 accesses, a row in registers (widths in multiples of 4 up to
// 4 * threads * LNV_MAX).
template <typename T, bool VEC>
__global__ void rmsnorm_add_norm_kernel(const float* __restrict__ y, const float* __restrict__ bias, const float* __restrict__ w,
                                        float* __restrict__ x, const float* __restrict__ w2, T* __restrict__ h, int H, float eps,
                                        float eps2) {
    ce_pdl_begin();
    __shared__ float scratch[32];
    const int t = blockIdx.x, tid = threadIdx.x;
    if (VEC) {
        const int H4 = H >> 2;
        const float4* yr = reinterpret_cast<const float4*>(y + (size_t)t * H);
        const float4* b4 = reinterpret_cast<const float4*>(bias);
        const float4* w4 = reinterpret_cast<const float4*>(w);
        float4* xr = reinterpret_cast<float4*>(x + (size_t)t * H);
        float4 v[LNV_MAX], xv[LNV_MAX];
        float q = 0.f;
#pragma unroll
        for (int n = 0; n < LNV_MAX; ++n) {
            int j = tid + n * blockDim.x;
            v[n] = j < H4 ? yr[j] : make_float4(0.f, 0.f, 0.f, 0.f);
            xv[n] = j < H4 ? xr[j] : make_float4(0.f, 0.f, 0.f, 0.f);
            if (bias && j < H4) { float4 b = b4[j]; v[n].x += b.x; v[n].y += b.y; v[n].z += b.z; v[n].w += b.w; }
            q += (v[n].x * v[n].x + v[n].y * v[n].y) + (v[n].z * v[n].z + v[n].w * v[n].w);
        }
        float inv = 1.0f / sqrtf(ce_block_sum(q, scratch) / (float)H + eps);
        q = 0.f;
#pragma unroll
        for (int n = 0; n < LNV_MAX; ++n) {
            int j = tid + n * blockDim.x;
            if (j < H4) {
                float4 ww = w4[j];
                xv[n].x += v[n].x * inv * ww.x; xv[n].y += v[n].y * inv * ww.y; xv[n].z += v[n].z * inv * ww.z; xv[n].w += v[n].w * inv * ww.w;
                xr[j] = xv[n];
            }
            q += (xv[n].x * xv[n].x + xv[n].y * xv[n].y) + (xv[n].z * xv[n].z + xv[n].w * xv[n].w);
        }
        if (!h) return;
        inv = 1.0f / sqrtf(ce_block_sum(q, scratch) / (float)H + eps2);
        const float4* w24 = reinterpret_cast<const float4*>(w2);
#pragma unroll
        for (int n = 0; n < LNV_MAX; ++n) {
            int j = tid + n * blockDim.x;
            if (j >= H4) continue;
            float4 ww = w24[j];
            float o0 = xv[n].x * inv * ww.x, o1 = xv[n].y * inv * ww.y, o2 = xv[n].z * inv * ww.z, o3 = xv[n].w * inv * ww.w;
            if (sizeof(T) == 4) reinterpret_cast<float4*>(h + (size_t)t * H)[j] = make_float4(o0, o1, o2, o3);
            else {
                __nv_bfloat162 lo = __floats2bfloat162_rn(o0, o1), hi = __floats2bfloat162_rn(o2, o3);
                reinterpret_cast<uint2*>(h + (size_t)t * H)[j] = make_uint2(*reinterpret_cast<unsigned*>(&lo), *reinterpret_cast<unsigned*>(&hi));
            }
        }
    } else {
        const float* yr = y + (size_t)t * H;
        float* xr = x + (size_t)t * H;
        float q = 0.f;
        for (int j = tid; j < H; j += blockDim.x) { float v = yr[j] + (bias ? bias[j] : 0.f); q = fmaf(v, v, q); }
        float inv = 1.0f / sqrtf(ce_block_sum(q, scratch) / (float)H + eps);
        q = 0.f;
        for (int j = tid; j < H; j += blockDim.x) {
            float v = xr[j] + (yr[j] + (bias ? bias[j] : 0.f)) * inv * w[j];
            xr[j] = v;
            q = fmaf(v, v, q);
        }
        if (!h) return;
        inv = 1.0f / sqrtf(ce_block_sum(q, scratch) / (float)H + eps2);
        for (int j = tid; j < H; j += blockDim.x) CeType<T>::store(h + (size_t)t * H + j, xr[j] * inv * w2[j]);       // (its own writes)
    }
}

extern "C" int ce_rmsnorm_add_norm(const float* y, const float* bias, const float* w, float* x, const float* w2, void* h, int h_dtype,
                                   int T, int H, float eps, float eps2, cudaStream_t stream) {
    if (T == 0) return CE_OK;
    if (!y || !w || !x || (h && !w2)) return ce_fail(CE_ERR_ARG, "ce_rmsnorm_add_norm: null pointer");
    if (H <= 0 || (h_dtype != CE_F32 && h_dtype != CE_BF16)) return ce_fail(CE_ERR_ARG, "ce_rmsnorm_add_norm: width %d, dtype %d", H, h_dtype);
    bool vec = H % 4 == 0 && H >= 256 && ((((uintptr_t)x | (uintptr_t)w | (uintptr_t)y | (uintptr_t)bias | (uintptr_t)w2 | (uintptr_t)h) & 15) == 0);
    int H4 = H / 4, vt = H4 >= 2048 ? 1024 : H4 >= 512 ? 512 : H4 >= 256 ? 256 : 128;
    ce_note("rmsnorm_add_norm_kernel");
    if (vec && H4 <= vt * LNV_MAX) {
        if (h_dtype == CE_F32) ce_launch(rmsnorm_add_norm_kernel<float, true>, T, vt, 0, stream, y, bias, w, x, w2, (float*)h, H, eps, eps2);
        else ce_launch(rmsnorm_add_norm_kernel<__nv_bfloat16, true>, T, vt, 0, stream, y, bias, w, x, w2, (__nv_bfloat16*)h, H, eps, eps2);
    } else {
        int th = H >= 4096 ? 512 : H >= 1024 ? 256 : 128;
        if (h_dtype == CE_F32) ce_launch(rmsnorm_add_norm_kernel<float, false>, T, th, 0, stream, y, bias, w, x, w2, (float*)h, H, eps, eps2);
        else ce_launch(rmsnorm_add_norm_kernel<__nv_bfloat16, false>, T, th, 0, stream, y, bias, w, x, w2, (__nv_bfloat16*)h, H, eps, eps2);
    }
    return ce_check_launch("ce_rmsnorm_add_norm");
}

// ---------------------------------------------------------------------------------------------
// The norm after the sum:  z = alpha x[t] + s,  x[t] = z / sqrt(mean(z^2) + eps) * w,  s the sublayer's output,
//   NM 0  y0[t] (+ bias), as it is
//   NM 3, 4  sum_k pick_w[t, k] rows[pair_row[t, k]], the weighted sum of a token's experts (rows float32 / bfloat16)
//   NM 1, 2  c * sum_m y_m[t] / sqrt(mean(y_m[t]^2) + eps_m) * w_m: the outputs of mixers side by side, each normed over the width
// store_only: s itself is stored in x (or, with alpha 1, added to it) and no norm is taken of the sum.
// xb (or null) receives the new x rounded to bfloat16.  VEC: float4 accesses, a row in registers.
// ---------------------------------------------------------------------------------------------
struct ResidualNormArgs {
    const float* y[2];
    const float* wm[2];          // the members' norm weights
    const float* bias;           // or null (NM 0)
    const float* w;              // null: store_only
    float* x;
    __nv_bfloat16* xb;
    int H;
    float alpha, c, eps, eps_m;
    const void* rows;            // NM 3, 4: [*, ld]
    const int* pair_row;         // [T, top]
    const float* pick_w;         // [T, top]
    int ld, top;
};

template <int NM, bool VEC>
__global__ void residual_norm_kernel(ResidualNormArgs a) {
    ce_pdl_begin();
    __shared__ float scratch[32];
    const int t = blockIdx.x, tid = threadIdx.x, H = a.H;
    constexpr bool PICKS = NM >= 3;
    constexpr int NY = NM == 2 ? 2 : 1;
    float inv_m[NY];
    if (VEC) {
        const int H4 = H >> 2;
        float4* xr = reinterpret_cast<float4*>(a.x + (size_t)t * H);
        float4 z[LNV_MAX], v[NY][LNV_MAX];
#pragma unroll
        for (int m = 0; m < NY; ++m)
#pragma unroll
            for (int n = 0; n < LNV_MAX; ++n) {
                int j = tid + n * blockDim.x;
                v[m][n] = make_float4(0.f, 0.f, 0.f, 0.f);
                if (j >= H4) continue;
                if (NM == 3) v[m][n] = ce_sum_picks4((const float*)a.rows, a.ld, a.pair_row + (size_t)t * a.top, a.pick_w + (size_t)t * a.top, a.top, 4 * j);
                else if (NM == 4) v[m][n] = ce_sum_picks4((const __nv_bfloat16*)a.rows, a.ld, a.pair_row + (size_t)t * a.top, a.pick_w + (size_t)t * a.top, a.top, 4 * j);
                else v[m][n] = reinterpret_cast<const float4*>(a.y[m] + (size_t)t * H)[j];
            }
#pragma unroll
        for (int n = 0; n < LNV_MAX; ++n) {
            int j = tid + n * blockDim.x;
            z[n] = j < H4 && a.alpha != 0.f ? xr[j] : make_float4(0.f, 0.f, 0.f, 0.f);
        }
        if (NM > 0 && !PICKS) {
#pragma unroll
            for (int m = 0; m < NY; ++m) {
                float q = 0.f;
#pragma unroll
                for (int n = 0; n < LNV_MAX; ++n) q += (v[m][n].x * v[m][n].x + v[m][n].y * v[m][n].y) + (v[m][n].z * v[m][n].z + v[m][n].w * v[m][n].w);
                inv_m[m] = 1.0f / sqrtf(ce_block_sum(q, scratch) / (float)H + a.eps_m);
            }
        }
        float q = 0.f;
#pragma unroll
        for (int n = 0; n < LNV_MAX; ++n) {
            int j = tid + n * blockDim.x;
            if (j >= H4) continue;
            float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
            if (NM == 0 || PICKS) {
                s = v[0][n];
                if (NM == 0 && a.bias) { float4 b = reinterpret_cast<const float4*>(a.bias)[j]; s.x += b.x; s.y += b.y; s.z += b.z; s.w += b.w; }
            } else {
#pragma unroll
                for (int m = 0; m < NY; ++m) {
                    float4 ww = reinterpret_cast<const float4*>(a.wm[m])[j];
                    s.x += v[m][n].x * inv_m[m] * ww.x; s.y += v[m][n].y * inv_m[m] * ww.y;
                    s.z += v[m][n].z * inv_m[m] * ww.z; s.w += v[m][n].w * inv_m[m] * ww.w;
                }
                s.x *= a.c; s.y *= a.c; s.z *= a.c; s.w *= a.c;
            }
            z[n].x = fmaf(a.alpha, z[n].x, s.x); z[n].y = fmaf(a.alpha, z[n].y, s.y);
            z[n].z = fmaf(a.alpha, z[n].z, s.z); z[n].w = fmaf(a.alpha, z[n].w, s.w);
            q += (z[n].x * z[n].x + z[n].y * z[n].y) + (z[n].z * z[n].z + z[n].w * z[n].w);
        }
        float inv = 1.0f;
        if (a.w) inv = 1.0f / sqrtf(ce_block_sum(q, scratch) / (float)H + a.eps);
#pragma unroll
        for (int n = 0; n < LNV_MAX; ++n) {
            int j = tid + n * blockDim.x;
            if (j >= H4) continue;
            if (a.w) {
                float4 ww = reinterpret_cast<const float4*>(a.w)[j];
                z[n].x *= inv * ww.x; z[n].y *= inv * ww.y; z[n].z *= inv * ww.z; z[n].w *= inv * ww.w;
            }
            xr[j] = z[n];
            if (a.xb) {
                __nv_bfloat162 lo = __floats2bfloat162_rn(z[n].x, z[n].y), hi = __floats2bfloat162_rn(z[n].z, z[n].w);
                reinterpret_cast<uint2*>(a.xb + (size_t)t * H)[j] = make_uint2(*reinterpret_cast<unsigned*>(&lo), *reinterpret_cast<unsigned*>(&hi));
            }
        }
    } else {
        float* xr = a.x + (size_t)t * H;
        if (NM > 0 && !PICKS) {
#pragma unroll
            for (int m = 0; m < NY; ++m) {
                float q = 0.f;
                for (int j = tid; j < H; j += blockDim.x) { float e = a.y[m][(size_t)t * H + j]; q = fmaf(e, e, q); }
                inv_m[m] = 1.0f / sqrtf(ce_block_sum(q, scratch) / (float)H + a.eps_m);
            }
        }
        float q = 0.f;
        for (int j = tid; j < H; j += blockDim.x) {
            float s = 0.f;
            if (NM == 0) s = a.y[0][(size_t)t * H + j] + (a.bias ? a.bias[j] : 0.f);
            else if (PICKS) {
                for (int k = 0; k < a.top; ++k) {
                    const size_t at = (size_t)a.pair_row[(size_t)t * a.top + k] * a.ld + j;
                    s = fmaf(a.pick_w[(size_t)t * a.top + k], NM == 3 ? ((const float*)a.rows)[at] : __bfloat162float(((const __nv_bfloat16*)a.rows)[at]), s);
                }
            } else {
#pragma unroll
                for (int m = 0; m < NY; ++m) s += a.y[m][(size_t)t * H + j] * inv_m[m] * a.wm[m][j];
                s *= a.c;
            }
            float z = a.alpha != 0.f ? fmaf(a.alpha, xr[j], s) : s;
            xr[j] = z;
            q = fmaf(z, z, q);
        }
        float inv = 1.0f;
        if (a.w) inv = 1.0f / sqrtf(ce_block_sum(q, scratch) / (float)H + a.eps);
        for (int j = tid; j < H; j += blockDim.x) {              // (its own writes)
            float z = a.w ? xr[j] * (inv * a.w[j]) : xr[j];
            xr[j] = z;
            if (a.xb) a.xb[(size_t)t * H + j] = __float2bfloat16_rn(z);
        }
    }
}

template <int NM>
static void residual_norm_launch(const ResidualNormArgs& a, int T, bool vec, cudaStream_t stream) {
    // Four float4s a thread: with fewer a block would take an SM's registers for threads that hold little of the row.  A bfloat16 step
    // of few tokens takes more threads a row instead, for its latency (in float32 the order of a row's sums must not depend on T).
    int H4 = a.H / 4, vt = H4 > 2048 ? 1024 : H4 > 1024 ? 512 : H4 > 512 ? 256 : 128;
    if (a.xb && T <= 64) vt = H4 >= 2048 ? 1024 : H4 >= 512 ? 512 : H4 >= 256 ? 256 : 128;
    if (vec && H4 <= vt * LNV_MAX) ce_launch(residual_norm_kernel<NM, true>, T, vt, 0, stream, a);
    else ce_launch(residual_norm_kernel<NM, false>, T, a.H >= 4096 ? 512 : a.H >= 1024 ? 256 : 128, 0, stream, a);
}

// members 0: y0 is the sublayer's output as it is (wm0, wm1, y1 null); 1 or 2: y0 (and y1) are normed with wm0 (wm1) and eps_m,
// their sum multiplied by c.  w null: the sum is stored without a norm (alpha 0: over what x held).
extern "C" int ce_residual_norm(const float* y0, const float* y1, const float* wm0, const float* wm1, int members, const float* bias,
                                const float* w, float* x, void* xb, int T, int H, float alpha, float c, float eps, float eps_m,
                                cudaStream_t stream) {
    if (T == 0) return CE_OK;
    if (!y0 || !x || members < 0 || members > 2 || (members > 0 && !wm0) || (members > 1 && (!wm1 || !y1)) || (members > 0 && bias))
        return ce_fail(CE_ERR_ARG, "ce_residual_norm: null pointer, or %d members", members);
    if (H <= 0) return ce_fail(CE_ERR_SIZE, "ce_residual_norm: width %d", H);
    ResidualNormArgs a{{y0, y1}, {wm0, wm1}, bias, w, x, (__nv_bfloat16*)xb, H, alpha, c, eps, eps_m, nullptr, nullptr, nullptr, 0, 0};
    bool vec = H % 4 == 0 && H >= 256 && ((((uintptr_t)y0 | (uintptr_t)y1 | (uintptr_t)wm0 | (uintptr_t)wm1 | (uintptr_t)bias |
                                            (uintptr_t)w | (uintptr_t)x | (uintptr_t)xb) & 15) == 0);
    ce_note("residual_norm_kernel");
    if (members == 0) residual_norm_launch<0>(a, T, vec, stream);
    else if (members == 1) residual_norm_launch<1>(a, T, vec, stream);
    else residual_norm_launch<2>(a, T, vec, stream);
    return ce_check_launch("ce_residual_norm");
}

// The same with the weighted sum of a token's experts as the sublayer's output: rows [*, ld] (float32 or bfloat16), pair_row and
// pick_w [T, top] as ce_moe_combine takes them.
extern "C" int ce_residual_norm_picks(const void* rows, int dtype, int ld, const int* pair_row, const float* pick_w, int top, const float* w,
                                      float* x, void* xb, int T, int H, float alpha, float eps, cudaStream_t stream) {
    if (T == 0) return CE_OK;
    if (!rows || !pair_row || !pick_w || !w || !x) return ce_fail(CE_ERR_ARG, "ce_residual_norm_picks: null pointer");
    if (H <= 0 || ld < H || top <= 0 || (dtype != CE_F32 && dtype != CE_BF16))
        return ce_fail(CE_ERR_SIZE, "ce_residual_norm_picks: width %d, rows of %d, %d picks, dtype %d", H, ld, top, dtype);
    ResidualNormArgs a{{nullptr, nullptr}, {nullptr, nullptr}, nullptr, w, x, (__nv_bfloat16*)xb, H, alpha, 1.0f, eps, 0.f, rows, pair_row, pick_w, ld, top};
    bool vec = H % 4 == 0 && ld % 4 == 0 && H >= 256 && ((((uintptr_t)rows | (uintptr_t)w | (uintptr_t)x | (uintptr_t)xb) & 15) == 0);
    ce_note("residual_norm_kernel (weighted sum of experts)");
    if (dtype == CE_F32) residual_norm_launch<3>(a, T, vec, stream);
    else residual_norm_launch<4>(a, T, vec, stream);
    return ce_check_launch("ce_residual_norm_picks");
}

// xb (or null): receives the new x rounded to bfloat16, what a sublayer that reads the residual itself takes as its input
extern "C" int ce_rmsnorm_add(const float* y, const float* w, float* x, void* xb, int T, int H, float eps, cudaStream_t stream) {
    if (T == 0) return CE_OK;
    if (!y || !w || !x) return ce_fail(CE_ERR_ARG, "ce_rmsnorm_add: null pointer");
    if (H % 4 == 0 && H >= 256 && ((((uintptr_t)x | (uintptr_t)w | (uintptr_t)y) & 15) == 0) && (((uintptr_t)xb) & 7) == 0) {
        int H4 = H / 4, vt = H4 >= 2048 ? 1024 : H4 >= 512 ? 512 : H4 >= 256 ? 256 : 128;
        if (H4 <= vt * LNV_MAX) {
            ce_note("rmsnorm_add_vec_kernel");
            ce_launch(rmsnorm_add_vec_kernel, T, vt, 0, stream, y, w, x, (__nv_bfloat16*)xb, H, eps);
            return ce_check_launch("ce_rmsnorm_add");
        }
    }
    ce_note("rmsnorm_add_kernel");
    ce_launch(rmsnorm_add_kernel, T, H >= 4096 ? 512 : H >= 1024 ? 256 : 128, 0, stream, y, w, x, (__nv_bfloat16*)xb, H, eps);
    return ce_check_launch("ce_rmsnorm_add");
}

// ---------------------------------------------------------------------------------------------
// x <- cap * tanh(x / cap), in place (the cap of the logits)
// ---------------------------------------------------------------------------------------------
__global__ void tanh_cap_kernel(float* __restrict__ x, size_t n, float cap, float inv_cap) {
    ce_pdl_begin();
    size_t stride = (size_t)gridDim.x * blockDim.x;
    for (size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x; e < n; e += stride) x[e] = cap * tanhf(x[e] * inv_cap);
}

extern "C" int ce_tanh_cap(float* x, long long n, float cap, cudaStream_t stream) {
    if (n == 0) return CE_OK;
    if (!x || !(cap > 0.f)) return ce_fail(CE_ERR_ARG, "ce_tanh_cap: null pointer or a cap that is not positive");
    long long blocks = (n + 255) / 256;
    if (blocks > 148 * 16) blocks = 148 * 16;
    ce_note("tanh_cap_kernel");
    ce_launch(tanh_cap_kernel, (int)blocks, 256, 0, stream, x, (size_t)n, cap, 1.0f / cap);
    return ce_check_launch("ce_tanh_cap");
}

// ---------------------------------------------------------------------------------------------
// out[t, l] = src[t, off + l] for l < L, rounded to the activation dtype: the input of a narrow second product
// ---------------------------------------------------------------------------------------------
template <typename T>
__global__ void copy_cols_kernel(const float* __restrict__ src, T* __restrict__ out, int ld, int off, int L, size_t total) {
    ce_pdl_begin();
    size_t stride = (size_t)gridDim.x * blockDim.x;
    for (size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += stride) {
        size_t t = e / L;
        int l = (int)(e % L);
        CeType<T>::store(out + e, src[t * ld + off + l]);
    }
}

extern "C" int ce_copy_cols(const float* src, void* out, int out_dtype, int T, int ld, int off, int L, cudaStream_t stream) {
    if (T == 0 || L == 0) return CE_OK;
    if (!src || !out) return ce_fail(CE_ERR_ARG, "ce_copy_cols: null pointer");
    size_t total = (size_t)T * L;
    size_t want = (total + 255) / 256;
    int blocks = (int)(want < (size_t)148 * 8 ? want : (size_t)148 * 8);
    ce_note("copy_cols_kernel");
    if (out_dtype == CE_F32) ce_launch(copy_cols_kernel<float>, blocks, 256, 0, stream, src, (float*)out, ld, off, L, total);
    else if (out_dtype == CE_BF16) ce_launch(copy_cols_kernel<__nv_bfloat16>, blocks, 256, 0, stream, src, (__nv_bfloat16*)out, ld, off, L, total);
    else return ce_fail(CE_ERR_ARG, "ce_copy_cols: unknown dtype %d", out_dtype);
    return ce_check_launch("ce_copy_cols");
}

// ---------------------------------------------------------------------------------------------
// Side input of a layer: g[t, j] = gelu_tanh(z[t, j]) * table[token[t], off + j]
// gelu_tanh(z) = 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3)))
// ---------------------------------------------------------------------------------------------
template <typename T>
__global__ void side_gate_kernel(const float* __restrict__ z, const T* __restrict__ table, const int* __restrict__ tokens,
                                 T* __restrict__ out, int D, int ld, int off, int V, int* __restrict__ status, size_t total) {
    ce_pdl_begin();
    size_t stride = (size_t)gridDim.x * blockDim.x;
    for (size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += stride) {
        size_t t = e / D;
        int j = (int)(e % D);
        int tok = tokens[t];
        float g = 0.f;
        if (tok < 0 || tok >= V) atomicExch(status, 1);
        else {
            float v = z[e];
            float inner = 0.79788456080286536f * (v + 0.044715f * v * v * v);
            g = 0.5f * v * (1.0f + tanhf(inner)) * CeType<T>::load(table + (size_t)tok * ld + off + j);
        }
        CeType<T>::store(out + e, g);
    }
}

extern "C" int ce_side_gate(const float* z, const void* table, int dtype, const int* tokens, void* out, int T, int D, int ld,
                            int off, int V, int* status, cudaStream_t stream) {
    if (T == 0 || D == 0) return CE_OK;
    if (!z || !table || !tokens || !out || !status) return ce_fail(CE_ERR_ARG, "ce_side_gate: null pointer");
    if (off < 0 || off + D > ld) return ce_fail(CE_ERR_SIZE, "ce_side_gate: columns %d..%d of a table %d wide", off, off + D, ld);
    size_t total = (size_t)T * D;
    size_t want = (total + 255) / 256;
    int blocks = (int)(want < (size_t)148 * 8 ? want : (size_t)148 * 8);
    ce_note("side_gate_kernel");
    if (dtype == CE_F32) ce_launch(side_gate_kernel<float>, blocks, 256, 0, stream, z, (const float*)table, tokens, (float*)out, D, ld, off, V, status, total);
    else if (dtype == CE_BF16) ce_launch(side_gate_kernel<__nv_bfloat16>, blocks, 256, 0, stream, z, (const __nv_bfloat16*)table, tokens, (__nv_bfloat16*)out, D, ld, off, V, status, total);
    else return ce_fail(CE_ERR_ARG, "ce_side_gate: unknown dtype %d", dtype);
    return ce_check_launch("ce_side_gate");
}
