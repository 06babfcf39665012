// Routed experts (mixture of experts): the choice of experts per token, the order of (token, choice) pairs by expert,
// the experts' products over the rows that chose them, and the weighted sum back into the token's stream.
//
//   z = W_router h (float32, a product of the caller);  the `top` largest z are chosen (ties: the lower index),
//   weights = softmax over the chosen z only;  out[t] += scale (sum_j weight_j * expert_{e_j}(h[t]) + sigmoid(g[t]) * shared(h[t])).
// Other scores, a correction of the choice, groups of experts and a factor on the weights: see k_route_topk and k_route_groups.
// The router may have more outputs than there are experts: the outputs from E on are identity experts, whose output is h[t]
// itself.  They take part in the choice, have no rows in the plan (pair_row -1), and the weighted sum adds weight * h[t] for them.
// An expert is a feed-forward: y = gate_act(W_gate h, W_up h), or act(W_up h) without a gate, then W_down y (see xr_gate below for the
// activations).  No step reads anything back to the host: the plan of who computes what is made on the device, and
// the grids are sized for the worst case (every tile index beyond the plan's count returns at once).
#include "common.cuh"
#include <math.h>

// ---------------------------------------------------------------------------------------------
// Choice: one warp per token.  ids [n][top] int32, wts [n][top] float32 (in the order of descending z).
// ---------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(128)
k_route_topk(const float* __restrict__ z, long long ldz, int* __restrict__ ids, float* __restrict__ wts, int n, int E, int top,
             const float* __restrict__ correction, int sigmoid_scores) {
    xr_pdl_launch();
    xr_pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t = blockIdx.x * 4 + warp;
    if (t >= n) return;
    const float* row = z + (size_t)t * ldz;
    float best0 = 0.f, sum = 0.f;
    int last_e = -1;
    float last_v = INFINITY;
    // the j-th choice: the largest value that comes after the (j-1)-th in the order (value descending, index ascending)
    for (int j = 0; j < top; j++) {
        float bv = -INFINITY;
        int be = 0x7fffffff;
        for (int e = lane; e < E; e += 32) {
            // (sigmoid scores: the choice is by score plus the expert's correction, where there is one)
            float v = row[e];
            if (sigmoid_scores) { v = 1.0f / (1.0f + expf(-v)); if (correction != nullptr) v += correction[e]; }
            const bool after = v < last_v || (v == last_v && e > last_e);
            if (after && (v > bv || (v == bv && e < be))) { bv = v; be = e; }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
            const int oe = __shfl_xor_sync(0xffffffffu, be, o);
            if (ov > bv || (ov == bv && oe < be)) { bv = ov; be = oe; }
        }
        if (j == 0) best0 = bv;
        // the weight: softmax over the chosen logits, or the chosen expert's score itself, without its correction
        const float p = sigmoid_scores ? 1.0f / (1.0f + expf(-row[be < E ? be : 0])) : expf(bv - best0);
        sum += p;
        if (lane == 0) { ids[(size_t)t * top + j] = be; wts[(size_t)t * top + j] = p; }
        last_v = bv; last_e = be;
    }
    __syncwarp();
    if (sigmoid_scores) return;
    if (lane < top) wts[(size_t)t * top + lane] /= sum;
    for (int j = 32 + lane; j < top; j += 32) wts[(size_t)t * top + j] /= sum;
}

// z: rows of E values, ldz apart.  sigmoid_scores: scores s = sigmoid(z); the `top` largest s + correction (correction [E] float32 or null) are chosen and their
// weights are s itself, not renormalised.  Otherwise the `top` largest z, weights their softmax.
XR_EXPORT int xr_route_topk(const float* z, long long ldz, int* ids, float* wts, int n, int E, int top, const float* correction, int sigmoid_scores,
                            cudaStream_t stream) {
    if (n < 1 || E < 1 || top < 1 || top > E || ldz < E || (correction != nullptr && !sigmoid_scores)) return XR_ERR_ARG;
    xr_launch(k_route_topk, dim3((n + 3) / 4), dim3(128), 0, stream, z, ldz, ids, wts, n, E, top, correction, sigmoid_scores ? 1 : 0);
    return xr_launch_status();
}

// ---------------------------------------------------------------------------------------------
// Choice with scores s = softmax(z) over ALL outputs and by groups: E outputs in `groups` equal groups of neighbours; the choice goes
// by c = s + correction (null: s); a group's score is its largest c, the `keep` best groups (ties: the lower index) stay and the
// `top` largest c inside them are chosen; weights s * scale, not renormalised.  One warp per token, c in shared memory.
// ---------------------------------------------------------------------------------------------
#define ROUTE_MAX_E 1024

__device__ __forceinline__ void route_argmax(float& v, int& i) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, v, o);
        const int oi = __shfl_xor_sync(0xffffffffu, i, o);
        if (ov > v || (ov == v && oi < i)) { v = ov; i = oi; }
    }
}

__global__ void __launch_bounds__(128)
k_route_groups(const float* __restrict__ z, int* __restrict__ ids, float* __restrict__ wts, int n, int E, int top,
               const float* __restrict__ correction, int groups, int keep, float scale) {
    xr_pdl_launch();
    extern __shared__ float route_sm[];                            // per warp: c [E], the groups' scores [groups], then the groups kept [groups]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x * 4 + warp, per = E / groups;
    if (t >= n) return;
    float* c = route_sm + (size_t)warp * (E + 2 * groups);
    float* best = c + E;
    float* stays = best + groups;
    xr_pdl_wait();
    const float* row = z + (size_t)t * E;
    float m = -INFINITY, sum = 0.f;
    for (int e = lane; e < E; e += 32) m = fmaxf(m, row[e]);
    m = xr_warp_max(m);
    for (int e = lane; e < E; e += 32) sum += expf(row[e] - m);
    sum = xr_warp_sum(sum);
    for (int e = lane; e < E; e += 32) c[e] = expf(row[e] - m) / sum + (correction != nullptr ? correction[e] : 0.f);
    __syncwarp();
    if (groups > 1) {
        for (int g = lane; g < groups; g += 32) {
            float b = -INFINITY;
            for (int e = g * per; e < (g + 1) * per; e++) b = fmaxf(b, c[e]);
            best[g] = b;
            stays[g] = 0.f;
        }
        __syncwarp();
        for (int k = 0; k < keep; k++) {
            float bv = -INFINITY;
            int bg = 0x7fffffff;
            for (int g = lane; g < groups; g += 32)
                if (stays[g] == 0.f && (bg == 0x7fffffff || best[g] > bv)) { bv = best[g]; bg = g; }
            route_argmax(bv, bg);
            if (lane == 0 && bg < groups) stays[bg] = 1.f;
            __syncwarp();
        }
        for (int e = lane; e < E; e += 32)
            if (stays[e / per] == 0.f) c[e] = -INFINITY;
        __syncwarp();
    }
    for (int j = 0; j < top; j++) {
        float bv = -INFINITY;
        int be = 0x7fffffff;
        for (int e = lane; e < E; e += 32)
            if (c[e] > bv) { bv = c[e]; be = e; }
        route_argmax(bv, be);
        if (be >= E) be = 0;                                       // (nothing left to choose: scores that are no numbers)
        if (lane == 0) {
            ids[(size_t)t * top + j] = be;
            wts[(size_t)t * top + j] = expf(row[be] - m) / sum * scale;
            c[be] = -INFINITY;
        }
        __syncwarp();
    }
}

// E: outputs of the router, identity experts included.  groups 1 (keep 1): no groups.
XR_EXPORT int xr_route_groups(const float* z, int* ids, float* wts, int n, int E, int top, const float* correction, int groups, int keep,
                              float scale, cudaStream_t stream) {
    if (n < 1 || E < 1 || E > ROUTE_MAX_E || groups < 1 || E % groups || keep < 1 || keep > groups || top < 1 || top > keep * (E / groups))
        return XR_ERR_ARG;
    const size_t smem = 4 * (size_t)(E + 2 * groups) * sizeof(float);
    if (smem > 48 * 1024) return XR_ERR_ARG;
    xr_launch(k_route_groups, dim3((n + 3) / 4), dim3(128), smem, stream, z, ids, wts, n, E, top, correction, groups, keep, scale);
    return xr_launch_status();
}

// ---------------------------------------------------------------------------------------------
// Plan, one block: rows = the n * top pairs sorted by expert, every expert's rows starting at a multiple of `align`
// (the row tile of the kernel that multiplies them), so that a tile of `align` rows meets one expert.
//   row_src [max_rows]: the pair (t * top + j) that row r computes, -1 for a row of padding;
//   pair_row [pairs]: the row of every pair;  tile_group [max_rows / align]: the tile's expert, -1 for a tile without rows.
//   max_rows = (pairs / align + E + 1) * align always suffices.  A pair whose id is E or more (an identity expert) has no row.
// Which row a pair gets among its expert's rows depends on the order in which threads arrive; a row's result does not.
// ---------------------------------------------------------------------------------------------
#define MOE_MAX_E 1024

__global__ void __launch_bounds__(1024)
k_moe_plan(const int* __restrict__ ids, int* __restrict__ row_src, int* __restrict__ pair_row, int* __restrict__ tile_group,
           int pairs, int E, int align, int max_tiles) {
    xr_pdl_launch();
    __shared__ int count[MOE_MAX_E], cursor[MOE_MAX_E], tile0[MOE_MAX_E + 1];
    for (int e = threadIdx.x; e < E; e += blockDim.x) count[e] = 0;
    xr_pdl_wait();
    __syncthreads();
    for (int p = threadIdx.x; p < pairs; p += blockDim.x) {
        const int e = ids[p];
        if (e < E) atomicAdd(&count[e], 1);
    }
    __syncthreads();
    if (threadIdx.x == 0) {
        int tiles = 0;
        for (int e = 0; e < E; e++) {
            tile0[e] = tiles; cursor[e] = tiles * align;
            tiles += (count[e] + align - 1) / align;
        }
        tile0[E] = tiles;
    }
    __syncthreads();
    const int used = tile0[E];
    for (int r = threadIdx.x; r < max_tiles * align; r += blockDim.x) row_src[r] = -1;
    for (int t = threadIdx.x; t < max_tiles; t += blockDim.x) tile_group[t] = -1;
    __syncthreads();
    for (int e = threadIdx.x; e < E; e += blockDim.x)
        for (int t = tile0[e]; t < tile0[e + 1]; t++) tile_group[t] = e;
    for (int p = threadIdx.x; p < pairs; p += blockDim.x) {
        const int e = ids[p];
        if (e >= E) { pair_row[p] = -1; continue; }
        const int r = atomicAdd(&cursor[e], 1);
        row_src[r] = p;
        pair_row[p] = r;
    }
    (void)used;
}

XR_EXPORT int xr_moe_plan(const int* ids, int* row_src, int* pair_row, int* tile_group, int pairs, int E, int align, int max_tiles,
                          cudaStream_t stream) {
    if (pairs < 1 || E < 1 || E > MOE_MAX_E || align < 1 || max_tiles < pairs / align + E) return XR_ERR_ARG;
    xr_launch(k_moe_plan, dim3(1), dim3(1024), 0, stream, ids, row_src, pair_row, tile_group, pairs, E, align, max_tiles);
    return xr_launch_status();
}

// ---------------------------------------------------------------------------------------------
// out[r] = h[row_src[r] / top] for the rows of tiles that hold any, zeros for rows of padding: the first product's
// input in the order of the plan, for the tensor-core product (which reads its rows through a tensor map).  T: what a thread moves at a
// time (an element, or 16 bytes of them; ldh and width are counted in it).
// ---------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
k_moe_gather(const T* __restrict__ h, long long ldh, T* __restrict__ out, const int* __restrict__ row_src,
             const int* __restrict__ tile_group, int top, int width, int align) {
    xr_pdl_launch();
    xr_pdl_wait();
    const int r = blockIdx.x;
    if (tile_group[r / align] < 0) return;
    const int src = row_src[r];
    T* o = out + (size_t)r * width;
    if (src < 0) {
        for (int i = threadIdx.x; i < width; i += blockDim.x) o[i] = T{};
        return;
    }
    const T* a = h + (size_t)(src / top) * ldh;
    for (int i = threadIdx.x; i < width; i += blockDim.x) o[i] = a[i];
}

XR_EXPORT int xr_moe_gather(const void* h, int dtype, long long ldh, void* out, const int* row_src, const int* tile_group, int top,
                            int width, int align, int max_rows, cudaStream_t stream) {
    if (max_rows < 1 || width < 1 || top < 1 || align < 1) return XR_ERR_ARG;
    if (dtype != XR_F32 && dtype != XR_BF16) return XR_ERR_ARG;
    const int size = dtype == XR_F32 ? 4 : 2, per = 16 / size;
#define GATHER(T, DIV)                                                                                                                       \
    do {                                                                                                                                     \
        const int units = width / (DIV), threads = units >= 256 ? 256 : (units + 31) / 32 * 32;                                              \
        xr_launch((k_moe_gather<T>), dim3(max_rows), dim3(threads), 0, stream, (const T*)h, ldh / (DIV), (T*)out, row_src, tile_group, top,  \
                  units, align);                                                                                                             \
    } while (0)
    if (width % per == 0 && ldh % per == 0 && !(((uintptr_t)h | (uintptr_t)out) & 15)) GATHER(uint4, per);
    else if (dtype == XR_F32) GATHER(float, 1);
    else GATHER(__nv_bfloat16, 1);
#undef GATHER
    return xr_launch_status();
}

// ---------------------------------------------------------------------------------------------
// The experts' products over the planned tiles (align = 64 rows), float32 FMA, k in ascending order for every result:
// the products of the true 32-bit path and of sizes the tensor-core product does not take.
//  first product (gated = 1): rows gather their token's h (row_src[r] / top); W = [E][2F][K] (an expert's gate rows,
//    then its up rows); out Y [rows][F] in the activation dtype = gate_act(h . w_gate_f, h . w_up_f).
//  first product of experts without a gate (gated = 0, gather = 1): W = [E][F][K]; out Y [rows][F] = act(h . w_f).
//  second product (gated = 0, gather = 0): rows read Y [rows][K = F]; W = [E][N][K]; out Z [rows][N] float32.
// Tile: 64 rows x 64 columns (gated: 32 features, gate and up side by side), 256 threads with 4 x 4 results each.
// ---------------------------------------------------------------------------------------------
#define MOE_TM 64
XR_EXPORT int xr_moe_tile_rows() { return MOE_TM; }

__device__ __forceinline__ float moe_gate(int act, float limit, float g, float u) {
    if (act == 3) {                  // g' sigmoid(1.702 g') (u' + 1), g' = min(g, limit), u' = clamp(u, -limit, limit)
        g = fminf(g, limit);
        u = fminf(fmaxf(u, -limit), limit);
        return g / (1.0f + expf(-1.702f * g)) * (u + 1.0f);
    }
    if (act == 1) return (g < -80.0f ? 0.0f : g / (1.0f + expf(-g))) * u;
    if (act == 2) return 0.5f * g * (1.0f + tanhf(0.7978845608f * (g + 0.044715f * g * g * g))) * u;
    if (act == 4) { const float r = fmaxf(g, 0.f); return r * r * u; }
    return g * u;
}

template <typename TA, typename TW, typename TO>
__global__ void __launch_bounds__(256)
k_moe_gemm(const TA* __restrict__ A, long long lda, const TW* __restrict__ W, TO* __restrict__ out, long long ldo,
           const int* __restrict__ row_src, const int* __restrict__ tile_group, int top, int N, int K, int gated, int gather, int act, float limit) {
    xr_pdl_launch();
    __shared__ float As[16][64 + 1], Ws[16][64 + 1];
    __shared__ int src_row[64];
    xr_pdl_wait();
    const int e = tile_group[blockIdx.x];
    if (e < 0) return;
    const int r0 = blockIdx.x * MOE_TM;
    const int cols = gated ? 32 : 64;                 // output columns (features) per tile
    const int c0 = blockIdx.y * cols;
    const TW* We = W + (size_t)e * (gated ? 2 : 1) * N * K;
    if (threadIdx.x < 64) {
        const int r = threadIdx.x, s = row_src[r0 + r];
        src_row[r] = s < 0 ? -1 : (gather ? s / top : r0 + r);
    }
    __syncthreads();
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < K; k0 += 16) {
        for (int i = threadIdx.x; i < 16 * 64; i += 256) {
            const int kk = i & 15, r = i >> 4, k = k0 + kk, s = src_row[r];
            As[kk][r] = (s >= 0 && k < K) ? xr_to_f32<TA>(A[(size_t)s * lda + k]) : 0.f;
        }
        for (int i = threadIdx.x; i < 16 * 64; i += 256) {
            const int kk = i & 15, c = i >> 4, k = k0 + kk;
            // gated: columns 0..31 are gate rows c0 + c, columns 32..63 the up rows of the same features
            const int wrow = gated ? (c < 32 ? c0 + c : N + c0 + c - 32) : c0 + c;
            const bool ok = k < K && (gated ? (c0 + (c & 31) < N) : (c0 + c < N));
            Ws[kk][c] = ok ? xr_to_f32<TW>(We[(size_t)wrow * K + k]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < 16; kk++) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; i++) { a[i] = As[kk][ty + 16 * i]; b[i] = Ws[kk][tx + 16 * i]; }
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const int r = ty + 16 * i;
        if (src_row[r] < 0) continue;
        TO* orow = out + (size_t)(r0 + r) * ldo;
        if (gated) {
            // this thread's columns tx, tx + 16 are gate sums, tx + 32, tx + 48 the up sums of the same two features
#pragma unroll
            for (int j = 0; j < 2; j++) {
                const int f = c0 + tx + 16 * j;
                if (f < N) orow[f] = xr_from_f32<TO>(moe_gate(act, limit, acc[i][j], acc[i][j + 2]));
            }
        } else {
#pragma unroll
            for (int j = 0; j < 4; j++) {
                const int c = c0 + tx + 16 * j;
                if (c < N) orow[c] = xr_from_f32<TO>(moe_gate(act, limit, acc[i][j], 1.0f));
            }
        }
    }
}

// a_dtype: of A; w_dtype: of the experts' matrices; max_tiles: tiles of 64 rows the plan may use.
XR_EXPORT int xr_moe_gemm(const void* A, int a_dtype, long long lda, const void* W, int w_dtype, void* out, int out_dtype,
                          long long ldo, const int* row_src, const int* tile_group, int max_tiles,
                          int top, int N, int K, int gated, int gather, int act, float limit, cudaStream_t stream) {
    if (max_tiles < 1 || N < 1 || K < 1 || top < 1 || act < 0 || act > 4 || (gated && !gather) || (!gated && act == 3)) return XR_ERR_ARG;
    const int cols = gated ? 32 : 64;
    dim3 grid(max_tiles, (N + cols - 1) / cols);
    if (grid.y > 65535) return XR_ERR_ARG;
    typedef __nv_bfloat16 bf;
#define MG(TA, TW, TO) xr_launch((k_moe_gemm<TA, TW, TO>), grid, dim3(256), 0, stream, (const TA*)A, lda, (const TW*)W, (TO*)out, ldo, \
                                 row_src, tile_group, top, N, K, gated, gather, act, limit)
    const int key = a_dtype * 4 + w_dtype * 2 + out_dtype;
    switch (key) {
        case XR_BF16 * 4 + XR_BF16 * 2 + XR_BF16: MG(bf, bf, bf); break;
        case XR_BF16 * 4 + XR_BF16 * 2 + XR_F32: MG(bf, bf, float); break;
        case XR_F32 * 4 + XR_BF16 * 2 + XR_F32: MG(float, bf, float); break;
        case XR_F32 * 4 + XR_F32 * 2 + XR_F32: MG(float, float, float); break;
        case XR_BF16 * 4 + XR_F32 * 2 + XR_BF16: MG(bf, float, bf); break;
        case XR_BF16 * 4 + XR_F32 * 2 + XR_F32: MG(bf, float, float); break;
        default: return XR_ERR_ARG;
    }
#undef MG
    return xr_launch_status();
}

// ---------------------------------------------------------------------------------------------
// d[t] += scale (sum_j wts[t][j] Z[pair_row[t * top + j]] + sigmoid(sg[t]) sum_s shared[s][t]), j and s ascending (float32).  A pair
// without a row (pair_row -1) is an identity expert's: its term is wts[t][j] * h[t].  `shared` (null: none): the shared expert's output,
// or the partial sums of its last product where that was cut along K.  With `nw` the row is then normed in passing:
// out[t] = d[t] / sqrt(mean(d[t]^2) + eps) * nw.  A block a token; a thread VEC consecutive columns at a time, its first CB_KEEP of
// them in registers between the two passes.
// ---------------------------------------------------------------------------------------------
#define CB_KEEP 4

struct CombineArgs {
    float* d; const float* Z; const float* wts; const int* pair_row;
    const void* h; long long ldh;
    const float* shared; int splits; const float* sg; long long ld_sg;
    float scale;
    const float* nw; void* out; float eps;
    int n, width, top;
};

template <int VEC> struct CombineVec { float v[VEC]; };
template <int VEC>
__device__ __forceinline__ CombineVec<VEC> cb_load(const float* p) {
    CombineVec<VEC> r;
    if constexpr (VEC == 4) { const float4 x = xr_ld_now4(reinterpret_cast<const float4*>(p)); r.v[0] = x.x; r.v[1] = x.y; r.v[2] = x.z; r.v[3] = x.w; }
    else r.v[0] = xr_ld_now(p);
    return r;
}
template <int VEC>
__device__ __forceinline__ void cb_store(float* p, const CombineVec<VEC>& r) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else *p = r.v[0];
}

template <typename TH, typename TO, int VEC>
__global__ void __launch_bounds__(1024)
k_moe_combine(CombineArgs a) {
    xr_pdl_launch();
    extern __shared__ float cb_sm[];                 // the token's weights [top], then its rows [top]
    __shared__ float scratch[33];
    const int t = blockIdx.x, units = a.width / VEC, top = a.top;
    int* rows = reinterpret_cast<int*>(cb_sm + top);
    xr_pdl_wait();
    for (int j = threadIdx.x; j < top; j += blockDim.x) { cb_sm[j] = a.wts[(size_t)t * top + j]; rows[j] = a.pair_row[(size_t)t * top + j]; }
    __syncthreads();
    const float gate = a.shared == nullptr ? 0.f : (a.sg == nullptr ? 1.0f : 1.0f / (1.0f + expf(-a.sg[(size_t)t * a.ld_sg])));
    float* drow = a.d + (size_t)t * a.width;
    auto value = [&](int u) {
        const int c = u * VEC;
        const CombineVec<VEC> old = cb_load<VEC>(drow + c);
        CombineVec<VEC> s;
#pragma unroll
        for (int i = 0; i < VEC; i++) s.v[i] = 0.f;
        // four rows' loads in flight together (a row that does not exist reads row 0 and counts nothing)
        for (int j0 = 0; j0 < top; j0 += 4) {
            CombineVec<VEC> z[4];
#pragma unroll
            for (int q = 0; q < 4; q++) {
                const int j = min(j0 + q, top - 1);
                z[q] = cb_load<VEC>(a.Z + (size_t)max(rows[j], 0) * a.width + c);
            }
#pragma unroll
            for (int q = 0; q < 4; q++)
#pragma unroll
                for (int i = 0; i < VEC; i++) xr_ld_fence(z[q].v[i]);
#pragma unroll
            for (int q = 0; q < 4; q++) {
                if (j0 + q >= top) continue;
                const bool has = rows[j0 + q] >= 0;
#pragma unroll
                for (int i = 0; i < VEC; i++) {
                    float v = has ? z[q].v[i] : 0.f;
                    if (!has && a.h != nullptr) v = xr_to_f32<TH>(((const TH*)a.h)[(size_t)t * a.ldh + c + i]);
                    s.v[i] = fmaf(cb_sm[j0 + q], v, s.v[i]);
                }
            }
        }
        if (a.shared != nullptr) {
            float sh[VEC];
#pragma unroll
            for (int i = 0; i < VEC; i++) sh[i] = 0.f;
            for (int s0 = 0; s0 < a.splits; s0 += 4) {
                CombineVec<VEC> z[4];
#pragma unroll
                for (int q = 0; q < 4; q++) z[q] = cb_load<VEC>(a.shared + ((size_t)min(s0 + q, a.splits - 1) * a.n + t) * a.width + c);
#pragma unroll
                for (int q = 0; q < 4; q++)
#pragma unroll
                    for (int i = 0; i < VEC; i++) xr_ld_fence(z[q].v[i]);
#pragma unroll
                for (int q = 0; q < 4; q++)
#pragma unroll
                    for (int i = 0; i < VEC; i++) sh[i] += s0 + q < a.splits ? z[q].v[i] : 0.f;
            }
#pragma unroll
            for (int i = 0; i < VEC; i++) s.v[i] = fmaf(gate, sh[i], s.v[i]);
        }
#pragma unroll
        for (int i = 0; i < VEC; i++) s.v[i] = fmaf(a.scale, s.v[i], old.v[i]);
        cb_store<VEC>(drow + c, s);
        return s;
    };
    CombineVec<VEC> keep[CB_KEEP];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < CB_KEEP; k++) {
        const int u = threadIdx.x + k * blockDim.x;
        if (u < units) {
            keep[k] = value(u);
#pragma unroll
            for (int i = 0; i < VEC; i++) ss = fmaf(keep[k].v[i], keep[k].v[i], ss);
        }
    }
    for (int u = threadIdx.x + CB_KEEP * blockDim.x; u < units; u += blockDim.x) {
        const CombineVec<VEC> v = value(u);
#pragma unroll
        for (int i = 0; i < VEC; i++) ss = fmaf(v.v[i], v.v[i], ss);
    }
    if (a.nw == nullptr) return;
    ss = xr_block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)a.width + a.eps);
    TO* orow = (TO*)a.out + (size_t)t * a.width;
    auto put = [&](int u, const CombineVec<VEC>& v) {
        alignas(16) TO w[VEC];
#pragma unroll
        for (int i = 0; i < VEC; i++) w[i] = xr_from_f32<TO>(v.v[i] * inv * a.nw[u * VEC + i]);
        if constexpr (VEC == 4) {
            if constexpr (sizeof(TO) == 4) *reinterpret_cast<float4*>(orow + u * 4) = *reinterpret_cast<float4*>(w);
            else *reinterpret_cast<uint2*>(orow + u * 4) = *reinterpret_cast<uint2*>(w);
        } else orow[u] = w[0];
    };
#pragma unroll
    for (int k = 0; k < CB_KEEP; k++) {
        const int u = threadIdx.x + k * blockDim.x;
        if (u < units) put(u, keep[k]);
    }
    for (int u = threadIdx.x + CB_KEEP * blockDim.x; u < units; u += blockDim.x) {         // (this thread's own stores)
        CombineVec<VEC> v;
#pragma unroll
        for (int i = 0; i < VEC; i++) v.v[i] = drow[u * VEC + i];
        put(u, v);
    }
}

// d [n][width] float32.  h [n][ldh] in h_dtype: what the experts read, for identity experts; null: there are none.  shared
// [splits][n][width] float32 with sg (n values, ld_sg apart; null: no gate); nw [width] with out [n][width] in out_dtype.
XR_EXPORT int xr_moe_combine(float* d, const float* Z, const float* wts, const int* pair_row, const void* h, int h_dtype, long long ldh,
                             const float* shared, int splits, const float* sg, long long ld_sg, float scale, const float* nw, void* out,
                             int out_dtype, float eps, int n, int width, int top, cudaStream_t stream) {
    if (n < 1 || width < 1 || top < 1 || top > 4096 || (h != nullptr && ldh < width) || (shared != nullptr && splits < 1) || (nw == nullptr) != (out == nullptr))
        return XR_ERR_ARG;
    if ((h != nullptr && h_dtype != XR_F32 && h_dtype != XR_BF16) || (out != nullptr && out_dtype != XR_F32 && out_dtype != XR_BF16)) return XR_ERR_ARG;
    CombineArgs a{d, Z, wts, pair_row, h, ldh, shared, splits, sg, ld_sg, scale, nw, out, eps, n, width, top};
    const bool vec = !(width & 3) && !(((uintptr_t)d | (uintptr_t)Z | (uintptr_t)shared | (uintptr_t)out) & 15);
    // (few tokens: nothing but a row's own threads hides its loads' latency)
    const int units = vec ? width / 4 : width, most = n <= xr_sm_count() ? 1024 : 256, threads = units >= most ? most : (units + 31) / 32 * 32;
    const size_t smem = (size_t)top * 8;
#define CB1(TH, TO, VEC) xr_launch((k_moe_combine<TH, TO, VEC>), dim3(n), dim3(threads), smem, stream, a)
#define CB(TH, TO)                                                                                                                           \
    do {                                                                                                                                     \
        if (vec) CB1(TH, TO, 4);                                                                                                             \
        else CB1(TH, TO, 1);                                                                                                                 \
    } while (0)
    const bool hb = h != nullptr && h_dtype == XR_BF16, ob = out != nullptr && out_dtype == XR_BF16;
    if (hb && ob) CB(__nv_bfloat16, __nv_bfloat16);
    else if (hb) CB(__nv_bfloat16, float);
    else if (ob) CB(float, __nv_bfloat16);
    else CB(float, float);
#undef CB
#undef CB1
    return xr_launch_status();
}
