// Mixture of experts: routing, the layout of a step's (token, expert) pairs by expert, the experts' two products as
// grouped products over that layout, and the weighted sum back into token order.
//
//   route    z [T, ld] float32 router logits (+ a bias per expert) -> s = softmax(z[:E]) or sigmoid(z[:E]), or, for a softmax over
//            the chosen logits only, s = exp(z - max z) and choice by z itself; choice scores c = s (+ a correction per expert);
//            experts in `groups` equal groups of neighbours, a group's score the largest c in it or the sum of its two largest,
//            only the best `keep` groups' experts eligible; the `top` eligible experts with the largest c are chosen
//            (ties: the lower index); weights s / (sum of the chosen s + 1e-20) * scale, or s * scale as they are.
//            Column E of z, where there is one, is the logit of a shared expert's gate: sgate[t] = sigmoid(z[t, E]).
//            In bfloat16, for routers of up to 128 rows, the product that gives z is part of the kernel.
//   align    the T*top pairs sorted by expert into rows of a padded layout: every expert's rows start at a multiple of
//            the tile height BM, so a tile of BM rows belongs to ONE expert.  row_token[p] is the token of row p (-1: a
//            padding row), pair_row[i] the row of pair i, tile_expert[j] the expert of tile j, n_tiles[0] their count.
//            Nothing of it reaches the host: the products launch a grid for the most tiles a step of that size can have,
//            and blocks past n_tiles leave at once, so a captured graph replays with any routing.
//   products out[p] = act(in[row p's token, or p] W[e]^T), e = tile_expert[p / BM]; act = none, relu^2, or a gated
//            activation of row pairs (rows 2j and 2j + 1 of W[e] are feature j's gate and up): the clamped one, or
//            silu(gate) up.  Every output element is a sum over k in a fixed order that depends on neither the row's place in
//            its tile nor on the other rows, so a token's result does not depend on the batch.  float32 FMA for any size and both dtypes;
//            bfloat16 on the tensor cores (wmma m16n16k16, float32 sums) for sizes in multiples of 16.
//   combine  y[t] (+)= sum_k weight[t, k] out[pair_row[t*top + k]] + sgate[t] shared[t], in the order of k, float32.
#include "common.cuh"
#include <mma.h>

#define MOE_MAX_EXPERTS 4096

// ---------------------------------------------------------------------------------------------
// routing: one warp a token
// ---------------------------------------------------------------------------------------------
struct MoeRouteArgs {
    const float* z;
    int* ids;           // [T, top]
    float* weights;     // [T, top]
    float* sgate;       // [T] or null
    int T, ld, E, top, groups, keep;
    float scale;
    const float* correction;     // [E] or null: added to the scores for the choice, not for the weights
    int scoring;                 // 0: softmax over the experts, 1: sigmoid, 2: softmax over the chosen logits
    int group_score;             // 0: a group's largest choice score, 1: the sum of its two largest
    int renormalize;             // 1: the weights are divided by the sum of the chosen scores
    const float* bias;           // [E] or null: added to the logits
};

__device__ __forceinline__ void moe_warp_argmax(float& v, int& i) {
    for (int o = 16; o > 0; o >>= 1) {
        float ov = __shfl_xor_sync(0xffffffffu, v, o);
        int oi = __shfl_xor_sync(0xffffffffu, i, o);
        if (ov > v || (ov == v && oi < i)) { v = ov; i = oi; }
    }
}

// One token, one warp.  zr: the token's logits; s, c, gs: E floats of shared memory each: the scores; the choice scores (a chosen
// or barred expert's becomes -inf); the groups' scores (a kept group's becomes +inf).
__device__ __forceinline__ void moe_route_token(const MoeRouteArgs& a, int t, int lane, const float* zr, float* s, float* c, float* gs) {
    for (int e = lane; e < a.E; e += 32) c[e] = a.bias ? zr[e] + a.bias[e] : zr[e];       // the logits (each lane its own experts')
    if (a.scoring != 1) {
        float mx = -INFINITY;
        for (int e = lane; e < a.E; e += 32) mx = fmaxf(mx, c[e]);
        for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        float sum = 0.f;
        for (int e = lane; e < a.E; e += 32) { float v = expf(c[e] - mx); s[e] = v; sum += v; }
        for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        const float inv = a.scoring == 0 ? 1.0f / sum : 1.0f;
        for (int e = lane; e < a.E; e += 32) s[e] *= inv;
    } else {
        for (int e = lane; e < a.E; e += 32) s[e] = 1.0f / (1.0f + expf(-c[e]));
    }
    if (a.scoring != 2)
        for (int e = lane; e < a.E; e += 32) c[e] = a.correction ? s[e] + a.correction[e] : s[e];
    __syncwarp();
    if (a.groups > 1 && a.keep < a.groups) {
        const int size = a.E / a.groups;
        for (int g = lane; g < a.groups; g += 32) {
            float best = -INFINITY, second = -INFINITY;
            for (int j = 0; j < size; ++j) {
                float v = c[g * size + j];
                second = fmaxf(second, fminf(v, best));
                best = fmaxf(best, v);
            }
            gs[g] = a.group_score == 1 && size > 1 ? best + second : best;
        }
        __syncwarp();
        for (int k = 0; k < a.keep; ++k) {
            float v = -INFINITY; int i = 0x7fffffff;
            for (int g = lane; g < a.groups; g += 32) if (gs[g] < INFINITY && gs[g] > v) { v = gs[g]; i = g; }
            moe_warp_argmax(v, i);
            if (lane == 0 && i < a.groups) gs[i] = INFINITY;
            __syncwarp();
        }
        for (int e = lane; e < a.E; e += 32) if (gs[e / size] < INFINITY) c[e] = -INFINITY;
        __syncwarp();
    }
    float total = 0.f, mine = 0.f;                           // lane k keeps the k-th pick (32 picks at a time)
    int mine_id = 0;
    for (int k0 = 0; k0 < a.top; k0 += 32) {
        const int n = min(32, a.top - k0);
        for (int k = 0; k < n; ++k) {
            float v = -INFINITY; int i = 0x7fffffff;
            for (int e = lane; e < a.E; e += 32) if (c[e] > v) { v = c[e]; i = e; }
            moe_warp_argmax(v, i);
            if (i >= a.E) i = k0 + k;                        // (only scores that are no numbers leave nothing to choose)
            const float w = s[i];
            if (lane == k) { mine = w; mine_id = i; }
            if (lane == 0) c[i] = -INFINITY;
            total += w;
            __syncwarp();
        }
        if (lane < n) {
            a.ids[(size_t)t * a.top + k0 + lane] = mine_id;
            a.weights[(size_t)t * a.top + k0 + lane] = mine;        // scaled below, once the sum is known
        }
    }
    __syncwarp();
    const float norm = a.renormalize ? a.scale / (total + 1e-20f) : a.scale;
    for (int k = lane; k < a.top; k += 32) a.weights[(size_t)t * a.top + k] *= norm;
    if (a.sgate && lane == 0) a.sgate[t] = 1.0f / (1.0f + expf(-zr[a.E]));
}

__global__ void __launch_bounds__(128) moe_route_kernel(MoeRouteArgs a) {
    ce_pdl_begin();
    extern __shared__ float moe_route_smem[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t = blockIdx.x * 4 + warp;
    if (t >= a.T) return;
    float* s = moe_route_smem + (size_t)warp * 3 * a.E;
    moe_route_token(a, t, lane, a.z + (size_t)t * a.ld, s, s + a.E, s + 2 * a.E);
}

// The router's product and the routing in one kernel (bfloat16): a block of 16 warps takes 16 tokens; the warps share K in runs of
// 32, each a product of the 16 tokens with all experts (mma.sync m16n8k16), and the partial logits are added in the warps' order
// (float32): a token's logits depend on neither its place nor on the other tokens.  Within a run the elements of K are dealt to the
// products so that every lane reads 16 consecutive bytes of a row (the same for both operands).  Then a warp routes a token.
// In a step of few tokens one block would read the whole router by itself: with CLUSTER > 1 that many blocks share K for the same 16
// tokens, and the first adds their logits up through distributed shared memory and routes.
#define MR_WARPS 16
__device__ __forceinline__ void moe_cluster_sync() {
    asm volatile("barrier.cluster.arrive.release.aligned;\nbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ float moe_ld_cluster(const float* mine, int rank) {
    unsigned at = (unsigned)__cvta_generic_to_shared(mine), there;
    float v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(there) : "r"(at), "r"(rank));
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(there) : "memory");
    return v;
}
struct MoeRouterArgs {
    const __nv_bfloat16* h;      // [T, ldh]
    const __nv_bfloat16* W;      // [N, K]: the experts' rows, then the shared expert's gate row where there is one
    int ldh, N, K;
};

template <int NT, int CLUSTER>
__global__ void __launch_bounds__(32 * MR_WARPS) moe_router_kernel(MoeRouterArgs r, MoeRouteArgs a) {
    ce_pdl_begin();
    extern __shared__ float moe_router_smem[];
    constexpr int NE = NT * 8;
    float* part = moe_router_smem;                           // [warps][16][NE]; the routing's work space afterwards
    float* z = part + MR_WARPS * 16 * NE;                    // [16][NE]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, grp = lane >> 2, quad = lane & 3;
    const int t0 = blockIdx.x / CLUSTER * 16, rank = blockIdx.x % CLUSTER;
    const __nv_bfloat16* ha = r.h + (size_t)min(t0 + grp, a.T - 1) * r.ldh + quad * 8;
    const __nv_bfloat16* hb = r.h + (size_t)min(t0 + grp + 8, a.T - 1) * r.ldh + quad * 8;
    float acc[NT][4];
#pragma unroll
    for (int n = 0; n < NT; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
#pragma unroll (NT >= 16 ? 1 : 4)
    for (int k0 = (rank * MR_WARPS + warp) * 32; k0 < r.K; k0 += CLUSTER * MR_WARPS * 32) {
        const uint4 x = *reinterpret_cast<const uint4*>(ha + k0), y = *reinterpret_cast<const uint4*>(hb + k0);
#pragma unroll
        for (int n = 0; n < NT; ++n) {
            const uint4 w = *reinterpret_cast<const uint4*>(r.W + (size_t)min(n * 8 + grp, r.N - 1) * r.K + quad * 8 + k0);
            asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                         : "+f"(acc[n][0]), "+f"(acc[n][1]), "+f"(acc[n][2]), "+f"(acc[n][3]) : "r"(x.x), "r"(y.x), "r"(x.y), "r"(y.y), "r"(w.x), "r"(w.y));
            asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                         : "+f"(acc[n][0]), "+f"(acc[n][1]), "+f"(acc[n][2]), "+f"(acc[n][3]) : "r"(x.z), "r"(y.z), "r"(x.w), "r"(y.w), "r"(w.z), "r"(w.w));
        }
    }
#pragma unroll
    for (int n = 0; n < NT; ++n) {
        float* p = part + (warp * 16 + grp) * NE + n * 8 + 2 * quad;
        p[0] = acc[n][0]; p[1] = acc[n][1];
        p[8 * NE] = acc[n][2]; p[8 * NE + 1] = acc[n][3];
    }
    __syncthreads();
    for (int e = threadIdx.x; e < 16 * NE; e += blockDim.x) {
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < MR_WARPS; ++w) v += part[w * 16 * NE + e];
        z[e] = v;
    }
    if (CLUSTER > 1) {
        moe_cluster_sync();                                  // every block's logits are there
        float* total = part;                                 // (its partial logits are used up)
        if (rank == 0)
            for (int e = threadIdx.x; e < 16 * NE; e += blockDim.x) {
                float v = z[e];
#pragma unroll
                for (int w = 1; w < CLUSTER; ++w) v += moe_ld_cluster(z + e, w);
                total[e] = v;
            }
        moe_cluster_sync();                                  // no block's shared memory goes away while it may still be read
        if (rank != 0) return;
        for (int e = threadIdx.x; e < 16 * NE; e += blockDim.x) z[e] = total[e];
    }
    __syncthreads();
    if (t0 + warp >= a.T) return;
    float* s = part + (size_t)warp * 3 * a.E;                // (16 warps x 3 E floats: less than the partial logits took)
    moe_route_token(a, t0 + warp, lane, z + warp * NE, s, s + a.E, s + 2 * a.E);
}

static int check_route(const char* who, const int* ids, const float* weights, int E, int top, int groups, int keep, int columns, bool gate,
                       const float* correction, int scoring, int group_score, int renormalize) {
    if (!ids || !weights) return ce_fail(CE_ERR_ARG, "%s: null pointer", who);
    if (E <= 0 || E > MOE_MAX_EXPERTS || top <= 0 || top > E || groups <= 0 || E % groups || keep <= 0 || keep > groups ||
        (long long)keep * (E / groups) < top || columns < E + (gate ? 1 : 0))
        return ce_fail(CE_ERR_SIZE, "%s: %d experts, top %d, %d groups of which %d are kept", who, E, top, groups, keep);
    if (scoring == 2 && (correction || !renormalize))
        return ce_fail(CE_ERR_ARG, "%s: a softmax over the chosen logits takes no correction and sums to the scale", who);
    if (scoring < 0 || scoring > 2 || group_score < 0 || group_score > 1)
        return ce_fail(CE_ERR_ARG, "%s: scoring %d, group score %d", who, scoring, group_score);
    return CE_OK;
}

extern "C" int ce_moe_route(const float* z, int* ids, float* weights, float* sgate, int T, int ld, int E, int top, int groups,
                            int keep, float scale, const float* correction, int scoring, int group_score, int renormalize,
                            const float* bias, cudaStream_t stream) {
    if (T == 0) return CE_OK;
    if (!z) return ce_fail(CE_ERR_ARG, "ce_moe_route: null pointer");
    int rc = check_route("ce_moe_route", ids, weights, E, top, groups, keep, ld, sgate != nullptr, correction, scoring, group_score, renormalize);
    if (rc) return rc;
    MoeRouteArgs a{z, ids, weights, sgate, T, ld, E, top, groups, keep, scale, correction, scoring, group_score, renormalize, bias};
    size_t smem = (size_t)4 * 3 * E * sizeof(float);
    if (smem > 40 * 1024) cudaFuncSetAttribute(moe_route_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    ce_note("moe_route_kernel");
    ce_launch(moe_route_kernel, (T + 3) / 4, 128, smem, stream, a);
    return ce_check_launch("ce_moe_route");
}

// rows of W (experts, and the gate) and elements of W that ce_moe_router takes: all of W passes through every block
extern "C" int ce_moe_router_supported(int N, int K, int ldh) {
    return N > 0 && N <= 128 && K >= 32 && K % 32 == 0 && ldh % 8 == 0 && (long long)N * K <= (1 << 20);
}

template <int NT>
static int moe_router_launch(const MoeRouterArgs& r, const MoeRouteArgs& a, cudaStream_t stream) {
    size_t smem = (size_t)(MR_WARPS + 1) * 16 * NT * 8 * sizeof(float);
    const int blocks = (a.T + 15) / 16;
    if (blocks > 8 || r.K < 4 * MR_WARPS * 32) {
        if (smem > 40 * 1024) cudaFuncSetAttribute(moe_router_kernel<NT, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        ce_launch(moe_router_kernel<NT, 1>, blocks, 32 * MR_WARPS, smem, stream, r, a);
        return ce_check_launch("ce_moe_router");
    }
    constexpr int CLUSTER = 8;
    if (smem > 40 * 1024) cudaFuncSetAttribute(moe_router_kernel<NT, CLUSTER>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(blocks * CLUSTER);
    cfg.blockDim = dim3(32 * MR_WARPS);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = CLUSTER; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = ce_pdl_enabled() ? 2 : 1;
    cudaError_t e = cudaLaunchKernelEx(&cfg, moe_router_kernel<NT, CLUSTER>, r, a);
    if (e != cudaSuccess) return ce_fail(CE_ERR_CUDA, "ce_moe_router: %s", cudaGetErrorString(e));
    return ce_check_launch("ce_moe_router");
}

// ce_moe_route with the router's product in the same kernel: h [T, ldh] bf16, W [>= N, K] bf16, N = E (+ 1 with sgate)
extern "C" int ce_moe_router(const void* h, int ldh, const void* W, int N, int K, int* ids, float* weights, float* sgate, int T, int E,
                             int top, int groups, int keep, float scale, const float* correction, int scoring, int group_score,
                             int renormalize, const float* bias, cudaStream_t stream) {
    if (T == 0) return CE_OK;
    if (!h || !W) return ce_fail(CE_ERR_ARG, "ce_moe_router: null pointer");
    if (!ce_moe_router_supported(N, K, ldh) || ldh < K || (((uintptr_t)h | (uintptr_t)W) & 15))
        return ce_fail(CE_ERR_SIZE, "ce_moe_router: %d rows of %d, row stride %d", N, K, ldh);
    int rc = check_route("ce_moe_router", ids, weights, E, top, groups, keep, N, sgate != nullptr, correction, scoring, group_score, renormalize);
    if (rc) return rc;
    MoeRouterArgs r{(const __nv_bfloat16*)h, (const __nv_bfloat16*)W, ldh, N, K};
    MoeRouteArgs a{nullptr, ids, weights, sgate, T, N, E, top, groups, keep, scale, correction, scoring, group_score, renormalize, bias};
    ce_note("moe_router_kernel");
    if (N <= 8) return moe_router_launch<1>(r, a, stream);
    if (N <= 16) return moe_router_launch<2>(r, a, stream);
    if (N <= 32) return moe_router_launch<4>(r, a, stream);
    if (N <= 64) return moe_router_launch<8>(r, a, stream);
    return moe_router_launch<16>(r, a, stream);
}

// ---------------------------------------------------------------------------------------------
// the pairs laid out by expert: one block
// ---------------------------------------------------------------------------------------------
// An expert's rows follow the order of the pairs.  Every warp owns a run of consecutive pairs: it counts them by expert, the
// warps' counts of an expert become the warps' first places by a running sum, and every warp deals its pairs out from there.
__global__ void __launch_bounds__(1024) moe_align_kernel(const int* __restrict__ ids, int n, int top, int E, int BM, int max_rows,
                                                         int* __restrict__ row_token, int* __restrict__ pair_row,
                                                         int* __restrict__ tile_expert, int* __restrict__ n_tiles) {
    ce_pdl_begin();
    extern __shared__ int moe_align_smem[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5;
    int* place = moe_align_smem;          // [n_warps][E]: a warp's count of an expert, then its next free row
    int* first = place + (size_t)n_warps * E;     // [E + 1]: an expert's first row
    for (int e = threadIdx.x; e < n_warps * E; e += blockDim.x) place[e] = 0;
    __syncthreads();
    const int per = ((n + n_warps - 1) / n_warps + 31) / 32 * 32;          // pairs a warp owns
    const int lo = min(n, warp * per), hi = min(n, lo + per);
    int* mine = place + (size_t)warp * E;
    for (int i = lo + lane; i < hi; i += 32) {
        int e = ids[i];
        if (e >= 0 && e < E) atomicAdd(&mine[e], 1);
    }
    __syncthreads();
    for (int e = threadIdx.x; e < E; e += blockDim.x) {           // the warps' counts to offsets within the expert
        int sum = 0;
        for (int w = 0; w < n_warps; ++w) {
            int c = place[(size_t)w * E + e];
            place[(size_t)w * E + e] = sum;
            sum += c;
        }
        first[e] = sum;
    }
    __syncthreads();
    if (threadIdx.x < 32) {               // a warp's running sum over the experts, 32 at a time
        int base = 0;
        for (int e0 = 0; e0 < E; e0 += 32) {
            int e = e0 + threadIdx.x;
            int c = e < E ? (first[e] + BM - 1) / BM * BM : 0, incl = c;
            for (int o = 1; o < 32; o <<= 1) {
                int v = __shfl_up_sync(0xffffffffu, incl, o);
                if ((int)threadIdx.x >= o) incl += v;
            }
            if (e < E) first[e] = base + incl - c;
            base += __shfl_sync(0xffffffffu, incl, 31);
        }
        if (threadIdx.x == 0) { first[E] = base; n_tiles[0] = base / BM; }
    }
    __syncthreads();
    const int rows = first[E];
    for (int p = threadIdx.x; p < rows && p < max_rows; p += blockDim.x) row_token[p] = -1;
    for (int e = threadIdx.x; e < E; e += blockDim.x)
        for (int p = first[e]; p < first[e + 1]; p += BM) tile_expert[p / BM] = e;
    __syncthreads();
    for (int i0 = lo; i0 < hi; i0 += 32) {
        const int i = i0 + lane, e = i < hi ? ids[i] : -1;
        const bool live = e >= 0 && e < E;
        const unsigned same = __match_any_sync(0xffffffffu, live ? e : -1);
        const int rank = __popc(same & ((1u << lane) - 1));
        int base = 0;
        if (live) base = mine[e];
        __syncwarp();
        if (live) {
            int p = first[e] + base + rank;
            pair_row[i] = p;
            row_token[p] = i / top;
            if (rank == __popc(same) - 1) mine[e] = base + rank + 1;
        }
        __syncwarp();
    }
}

extern "C" int ce_moe_max_tiles(int n_pairs, int E, int BM) {
    int busy = n_pairs < E ? n_pairs : E;                   // experts that can have a part-filled tile
    return n_pairs / BM + busy;
}

extern "C" int ce_moe_align(const int* ids, int n_pairs, int top, int E, int BM, int max_rows, int* row_token, int* pair_row,
                            int* tile_expert, int* n_tiles, cudaStream_t stream) {
    if (n_pairs == 0) return CE_OK;
    if (!ids || !row_token || !pair_row || !tile_expert || !n_tiles) return ce_fail(CE_ERR_ARG, "ce_moe_align: null pointer");
    if (E <= 0 || E > MOE_MAX_EXPERTS || BM <= 0 || top <= 0 || max_rows < ce_moe_max_tiles(n_pairs, E, BM) * BM)
        return ce_fail(CE_ERR_SIZE, "ce_moe_align: %d experts, tiles of %d, room for %d rows", E, BM, max_rows);
    int threads = n_pairs >= 1024 ? 1024 : (n_pairs + 31) / 32 * 32;
    while (threads > 32 && (size_t)(threads / 32 + 1) * E * sizeof(int) > 160 * 1024) threads /= 2;      // (many experts: fewer warps)
    threads = threads / 32 * 32;
    size_t smem = ((size_t)(threads / 32 + 1) * E + 1) * sizeof(int);
    if (smem > 40 * 1024) cudaFuncSetAttribute(moe_align_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    ce_note("moe_align_kernel");
    ce_launch(moe_align_kernel, 1, threads, smem, stream, ids, n_pairs, top, E, BM, max_rows, row_token, pair_row, tile_expert, n_tiles);
    return ce_check_launch("ce_moe_align");
}

// ---------------------------------------------------------------------------------------------
// grouped products
// ---------------------------------------------------------------------------------------------
enum { MOE_ACT_NONE = 0, MOE_ACT_RELU2 = 1, MOE_ACT_CLAMPGLU = 2, MOE_ACT_SILUGLU = 3 };      // 2, 3: of row pairs (gate, up), one output a pair
#define MOE_GATED(act) ((act) == MOE_ACT_CLAMPGLU || (act) == MOE_ACT_SILUGLU)

__device__ __forceinline__ float moe_act(int act, float v) {
    if (act == MOE_ACT_RELU2) { v = fmaxf(v, 0.f); return v * v; }
    return v;
}

struct MoeMatmulArgs {
    const void* in;              // [*, ldi]: row p's input is row row_token[p] (gather) or row p
    const void* W;               // [E, N, K]
    void* out;                   // [rows, ldo]
    const int* row_token;        // or null: rows are taken as they lie
    const int* tile_expert;
    const int* n_tiles;          // or null: every tile of the grid
    int ldi, ldo, N, K, BM, act, n_rows;     // n_rows: rows of `in` when they are taken as they lie (later rows are padding)
    float limit, alpha;          // the clamped activation's
};

#define MP_BN 64
#define MP_BK 16

// float32 FMA: a block of 256 threads takes BM (16 or 64) rows x 64 outputs; a thread (BM / 16) x 4 of them
template <typename T, int BM>
__global__ void __launch_bounds__(256) moe_matmul_plain_kernel(MoeMatmulArgs a) {
    ce_pdl_begin();
    const int tile = blockIdx.y;
    if (a.n_tiles && tile >= a.n_tiles[0]) return;
    constexpr int RPT = BM / 16;
    __shared__ float As[MP_BK][BM + 1];
    __shared__ float Ws[MP_BK][MP_BN + 1];
    __shared__ int src[BM];
    const int tid = threadIdx.x, n0 = blockIdx.x * MP_BN, p0 = tile * BM;
    const T* W = (const T*)a.W + (size_t)(a.tile_expert ? a.tile_expert[tile] : 0) * a.N * a.K;
    if (tid < BM) src[tid] = a.row_token ? a.row_token[p0 + tid] : (p0 + tid < a.n_rows ? p0 + tid : -1);
    __syncthreads();
    const int tm = (tid / 16) * RPT, tn = (tid % 16) * 4;
    float acc[RPT][4];
#pragma unroll
    for (int i = 0; i < RPT; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    for (int k0 = 0; k0 < a.K; k0 += MP_BK) {
        for (int e = tid; e < BM * MP_BK; e += 256) {
            int r = e / MP_BK, c = e % MP_BK, row = src[r];
            As[c][r] = (row >= 0 && k0 + c < a.K) ? CeType<T>::load((const T*)a.in + (size_t)row * a.ldi + k0 + c) : 0.f;
        }
        for (int e = tid; e < MP_BN * MP_BK; e += 256) {
            int r = e / MP_BK, c = e % MP_BK;
            Ws[c][r] = (n0 + r < a.N && k0 + c < a.K) ? CeType<T>::load(W + (size_t)(n0 + r) * a.K + k0 + c) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < MP_BK; ++kk) {
            float wv[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) wv[j] = Ws[kk][tn + j];
#pragma unroll
            for (int i = 0; i < RPT; ++i) {
                float av = As[kk][tm + i];
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av, wv[j], acc[i][j]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        if (src[tm + i] < 0) continue;
        if (MOE_GATED(a.act)) {
#pragma unroll
            for (int j = 0; j < 4; j += 2)
                if (n0 + tn + j < a.N)
                    CeType<T>::store((T*)a.out + (size_t)(p0 + tm + i) * a.ldo + (n0 + tn + j) / 2,
                                     a.act == MOE_ACT_SILUGLU ? ce_silu_glu(acc[i][j], acc[i][j + 1])
                                                              : ce_clamp_glu(acc[i][j], acc[i][j + 1], a.limit, a.alpha));
            continue;
        }
#pragma unroll
        for (int j = 0; j < 4; ++j)
            if (n0 + tn + j < a.N) CeType<T>::store((T*)a.out + (size_t)(p0 + tm + i) * a.ldo + n0 + tn + j, moe_act(a.act, acc[i][j]));
    }
}

// bfloat16 on the tensor cores: four warps; with tiles of 64 rows a warp takes 16 rows x 64 outputs, with tiles of 16 rows
// the warps take the four 16-column parts of the 64 outputs for the same rows.  The rows go through shared memory 64
// elements of K at a time; the weights' fragments come straight from memory (W[e] is [N, K] row-major: K x N column-major).
#define MW_BN 64
#define MW_BK 64

template <int BM>
__global__ void __launch_bounds__(128) moe_matmul_wmma_kernel(MoeMatmulArgs a) {
    using namespace nvcuda;
    ce_pdl_begin();
    const int tile = blockIdx.y;
    if (a.n_tiles && tile >= a.n_tiles[0]) return;
    constexpr bool FEW = BM == 16;
    __shared__ __align__(32) __nv_bfloat16 As[BM][MW_BK + 16];
    __shared__ __align__(32) float Cs[BM][MW_BN + 8];
    __shared__ int src[BM];
    const int tid = threadIdx.x, warp = tid >> 5, n0 = blockIdx.x * MW_BN, p0 = tile * BM;
    const __nv_bfloat16* W = (const __nv_bfloat16*)a.W + (size_t)(a.tile_expert ? a.tile_expert[tile] : 0) * a.N * a.K;
    const __nv_bfloat16* in = (const __nv_bfloat16*)a.in;
    if (tid < BM) src[tid] = a.row_token ? a.row_token[p0 + tid] : (p0 + tid < a.n_rows ? p0 + tid : -1);
    __syncthreads();
    const int n_frag = min(MW_BN, a.N - n0) / 16;
    constexpr int NF = FEW ? 1 : MW_BN / 16;
    const int wrow = FEW ? 0 : warp * 16, f0 = FEW ? warp : 0;
    wmma::fragment<wmma::accumulator, 16, 16, 16, float> acc[NF];
#pragma unroll
    for (int j = 0; j < NF; ++j) wmma::fill_fragment(acc[j], 0.f);
    for (int k0 = 0; k0 < a.K; k0 += MW_BK) {
        const int kw = min(MW_BK, a.K - k0);
        for (int e = tid; e < BM * (MW_BK / 8); e += 128) {
            int r = e / (MW_BK / 8), c = (e % (MW_BK / 8)) * 8, row = src[r];
            uint4 v = make_uint4(0u, 0u, 0u, 0u);
            if (row >= 0 && c < kw) v = *reinterpret_cast<const uint4*>(in + (size_t)row * a.ldi + k0 + c);
            *reinterpret_cast<uint4*>(&As[r][c]) = v;
        }
        __syncthreads();
        for (int kk = 0; kk < kw; kk += 16) {
            wmma::fragment<wmma::matrix_a, 16, 16, 16, __nv_bfloat16, wmma::row_major> fa;
            wmma::load_matrix_sync(fa, &As[wrow][kk], MW_BK + 16);
#pragma unroll
            for (int j = 0; j < NF; ++j) {
                if (f0 + j < n_frag) {
                    wmma::fragment<wmma::matrix_b, 16, 16, 16, __nv_bfloat16, wmma::col_major> fb;
                    wmma::load_matrix_sync(fb, W + (size_t)(n0 + (f0 + j) * 16) * a.K + k0 + kk, a.K);
                    wmma::mma_sync(acc[j], fa, fb, acc[j]);
                }
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int j = 0; j < NF; ++j)
        if (f0 + j < n_frag) wmma::store_matrix_sync(&Cs[wrow][(f0 + j) * 16], acc[j], MW_BN + 8, wmma::mem_row_major);
    __syncthreads();
    for (int e = tid; e < BM * (MW_BN / 2); e += 128) {
        int r = e / (MW_BN / 2), c = (e % (MW_BN / 2)) * 2;
        if (src[r] < 0 || n0 + c >= a.N) continue;
        if (MOE_GATED(a.act)) {
            ((__nv_bfloat16*)a.out)[(size_t)(p0 + r) * a.ldo + (n0 + c) / 2] =
                __float2bfloat16_rn(a.act == MOE_ACT_SILUGLU ? ce_silu_glu_fast(Cs[r][c], Cs[r][c + 1])
                                                             : ce_clamp_glu_fast(Cs[r][c], Cs[r][c + 1], a.limit, a.alpha));
            continue;
        }
        __nv_bfloat162 v = __floats2bfloat162_rn(moe_act(a.act, Cs[r][c]), moe_act(a.act, Cs[r][c + 1]));
        *reinterpret_cast<__nv_bfloat162*>((__nv_bfloat16*)a.out + (size_t)(p0 + r) * a.ldo + n0 + c) = v;
    }
}

// in [*, ldi], W [E, N, K], out [max_tiles * BM, ldo] (N columns, N / 2 with the activation of row pairs); BM is 16 or 64 and is the tile height the layout was made with.
// Without the layout's tables (all three null) it is one expert's product over n_rows rows as they lie.
extern "C" int ce_moe_matmul(const void* in, const void* W, void* out, const int* row_token, const int* tile_expert,
                             const int* n_tiles, int dtype, int max_tiles, int BM, int N, int K, int ldi, int ldo, int act,
                             float limit, float alpha, int n_rows, cudaStream_t stream) {
    if (max_tiles == 0 || N == 0) return CE_OK;
    if (!in || !W || !out || K <= 0) return ce_fail(CE_ERR_ARG, "ce_moe_matmul: null pointer or K=%d", K);
    if ((BM != 16 && BM != 64) || max_tiles > 65535) return ce_fail(CE_ERR_SIZE, "ce_moe_matmul: tiles of %d rows, %d tiles", BM, max_tiles);
    if (act < 0 || act > 3 || (MOE_GATED(act) && N % 2)) return ce_fail(CE_ERR_ARG, "ce_moe_matmul: activation %d of %d rows", act, N);
    MoeMatmulArgs a{in, W, out, row_token, tile_expert, n_tiles, ldi, ldo, N, K, BM, act, n_rows, limit, alpha};
    if (dtype == CE_BF16 && N % 16 == 0 && K % 16 == 0 && ldi % 8 == 0 && ldo % 2 == 0 &&
        ((((uintptr_t)in) & 15) == 0) && ((((uintptr_t)W) & 31) == 0) && ((((uintptr_t)out) & 3) == 0)) {
        dim3 grid((N + MW_BN - 1) / MW_BN, max_tiles);
        ce_note("moe_matmul_wmma_kernel");
        if (BM == 16) ce_launch(moe_matmul_wmma_kernel<16>, grid, 128, 0, stream, a);
        else ce_launch(moe_matmul_wmma_kernel<64>, grid, 128, 0, stream, a);
        return ce_check_launch("ce_moe_matmul");
    }
    dim3 grid((N + MP_BN - 1) / MP_BN, max_tiles);
    ce_note("moe_matmul_plain_kernel");
    if (dtype == CE_F32 && BM == 16) ce_launch(moe_matmul_plain_kernel<float, 16>, grid, 256, 0, stream, a);
    else if (dtype == CE_F32) ce_launch(moe_matmul_plain_kernel<float, 64>, grid, 256, 0, stream, a);
    else if (dtype == CE_BF16 && BM == 16) ce_launch(moe_matmul_plain_kernel<__nv_bfloat16, 16>, grid, 256, 0, stream, a);
    else if (dtype == CE_BF16) ce_launch(moe_matmul_plain_kernel<__nv_bfloat16, 64>, grid, 256, 0, stream, a);
    else return ce_fail(CE_ERR_ARG, "ce_moe_matmul: unknown dtype %d", dtype);
    return ce_check_launch("ce_moe_matmul");
}

// ---------------------------------------------------------------------------------------------
// the tokens' rows copied into the layout's order (what a product that loads its rows by TMA reads): row p of the
// live tiles receives row row_token[p] of the input, zeros where p is padding.  Rows are copied 16 bytes a thread.
// ---------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256) moe_gather_kernel(const uint4* __restrict__ in, long long ldi16, const int* __restrict__ row_token,
                                                         const int* __restrict__ n_tiles, int BM, uint4* __restrict__ out, int row16,
                                                         int max_rows) {
    ce_pdl_begin();
    const int rows = min(n_tiles[0] * BM, max_rows);
    const int per = blockDim.x / row16 > 0 ? blockDim.x / row16 : 1;          // rows a block copies at a time
    for (int p0 = blockIdx.x * per; p0 < rows; p0 += gridDim.x * per) {
        if (row16 <= (int)blockDim.x) {
            int p = p0 + threadIdx.x / row16, j = threadIdx.x % row16;
            if (threadIdx.x < per * row16 && p < rows) {
                int t = row_token[p];
                out[(size_t)p * row16 + j] = t >= 0 ? in[(size_t)t * ldi16 + j] : make_uint4(0, 0, 0, 0);
            }
        } else {
            int t = row_token[p0];
            for (int j = threadIdx.x; j < row16; j += blockDim.x)
                out[(size_t)p0 * row16 + j] = t >= 0 ? in[(size_t)t * ldi16 + j] : make_uint4(0, 0, 0, 0);
        }
    }
}

// in [T, ldi] -> out [max_rows, K] (contiguous), elements of `elsize` bytes; K * elsize and ldi * elsize multiples of 16
extern "C" int ce_moe_gather(const void* in, int ldi, int K, int elsize, const int* row_token, const int* n_tiles, int BM, void* out,
                             int max_rows, cudaStream_t stream) {
    if (max_rows == 0 || K == 0) return CE_OK;
    if (!in || !row_token || !n_tiles || !out) return ce_fail(CE_ERR_ARG, "ce_moe_gather: null pointer");
    if (((long long)K * elsize) % 16 || ((long long)ldi * elsize) % 16 || (((uintptr_t)in | (uintptr_t)out) & 15) || BM <= 0)
        return ce_fail(CE_ERR_SIZE, "ce_moe_gather: rows of %d elements of %d bytes are not whole 16-byte pieces", K, elsize);
    int row16 = (int)((long long)K * elsize / 16);
    int per = 256 / row16 > 0 ? 256 / row16 : 1;
    int blocks = (max_rows + per - 1) / per;
    int cap = ce_sm_count() * 8;
    if (blocks > cap) blocks = cap;
    ce_note("moe_gather_kernel");
    ce_launch(moe_gather_kernel, blocks, 256, 0, stream, (const uint4*)in, (long long)ldi * elsize / 16, row_token, n_tiles, BM, (uint4*)out,
              row16, max_rows);
    return ce_check_launch("ce_moe_gather");
}

// ---------------------------------------------------------------------------------------------
// back to token order
// ---------------------------------------------------------------------------------------------
template <typename T>
__global__ void moe_combine_kernel(const T* __restrict__ rows, int ld, const int* __restrict__ pair_row, const float* __restrict__ weights,
                                   const T* __restrict__ shared, const float* __restrict__ sgate, float* __restrict__ y, int top,
                                   int W, int accumulate) {
    ce_pdl_begin();
    const int t = blockIdx.x;
    for (int j = blockIdx.y * blockDim.x + threadIdx.x; j < W; j += blockDim.x * gridDim.y) {
        float v = 0.f;
        for (int k = 0; k < top; ++k)
            v = fmaf(weights[(size_t)t * top + k], CeType<T>::load(rows + (size_t)pair_row[(size_t)t * top + k] * ld + j), v);
        if (shared) v = fmaf(sgate ? sgate[t] : 1.0f, CeType<T>::load(shared + (size_t)t * W + j), v);
        float* o = y + (size_t)t * W + j;
        *o = accumulate ? *o + v : v;
    }
}

// The same with four columns a thread (W and ld in multiples of 4, rows aligned): the same sums in the same order.
template <typename T>
__global__ void moe_combine_vec_kernel(const T* __restrict__ rows, int ld, const int* __restrict__ pair_row, const float* __restrict__ weights,
                                       const T* __restrict__ shared, const float* __restrict__ sgate, float* __restrict__ y, int top,
                                       int W, int accumulate) {
    ce_pdl_begin();
    const int t = blockIdx.x;
    const int j = 4 * (blockIdx.y * blockDim.x + threadIdx.x);
    if (j >= W) return;
    float4 v = ce_sum_picks4(rows, ld, pair_row + (size_t)t * top, weights + (size_t)t * top, top, j);
    if (shared) {
        const float g = sgate ? sgate[t] : 1.0f;
        const float4 s = ce_load4(shared + (size_t)t * W + j);
        v.x = fmaf(g, s.x, v.x); v.y = fmaf(g, s.y, v.y); v.z = fmaf(g, s.z, v.z); v.w = fmaf(g, s.w, v.w);
    }
    float4* o = reinterpret_cast<float4*>(y + (size_t)t * W + j);
    if (accumulate) { const float4 p = *o; v.x = p.x + v.x; v.y = p.y + v.y; v.z = p.z + v.z; v.w = p.w + v.w; }
    *o = v;
}

extern "C" int ce_moe_combine(const void* rows, int dtype, int ld, const int* pair_row, const float* weights, const void* shared,
                              const float* sgate, float* y, int T, int top, int W, int accumulate, cudaStream_t stream) {
    if (T == 0 || W == 0) return CE_OK;
    if (!rows || !pair_row || !weights || !y) return ce_fail(CE_ERR_ARG, "ce_moe_combine: null pointer");
    const size_t el = dtype == CE_F32 ? 4 : 2;
    const int threads = 128;
    ce_note("moe_combine_kernel");
    if (W % 4 == 0 && ld % 4 == 0 && ((uintptr_t)y & 15) == 0 && (((uintptr_t)rows | (uintptr_t)shared) & (4 * el - 1)) == 0) {
        dim3 grid(T, (W / 4 + threads - 1) / threads);
        if (dtype == CE_F32) ce_launch(moe_combine_vec_kernel<float>, grid, threads, 0, stream, (const float*)rows, ld, pair_row, weights, (const float*)shared, sgate, y, top, W, accumulate);
        else if (dtype == CE_BF16) ce_launch(moe_combine_vec_kernel<__nv_bfloat16>, grid, threads, 0, stream, (const __nv_bfloat16*)rows, ld, pair_row, weights, (const __nv_bfloat16*)shared, sgate, y, top, W, accumulate);
        else return ce_fail(CE_ERR_ARG, "ce_moe_combine: unknown dtype %d", dtype);
        return ce_check_launch("ce_moe_combine");
    }
    dim3 grid(T, (W + 4 * threads - 1) / (4 * threads));
    if (dtype == CE_F32) ce_launch(moe_combine_kernel<float>, grid, threads, 0, stream, (const float*)rows, ld, pair_row, weights, (const float*)shared, sgate, y, top, W, accumulate);
    else if (dtype == CE_BF16) ce_launch(moe_combine_kernel<__nv_bfloat16>, grid, threads, 0, stream, (const __nv_bfloat16*)rows, ld, pair_row, weights, (const __nv_bfloat16*)shared, sgate, y, top, W, accumulate);
    else return ce_fail(CE_ERR_ARG, "ce_moe_combine: unknown dtype %d", dtype);
    return ce_check_launch("ce_moe_combine");
}
