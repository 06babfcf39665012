// Linear recurrences with a fixed-size float32 state per request slot.
//
// (1) The real-gated linear recurrent unit (the recurrence of Griffin's recurrent block).  With R channels in B blocks of
//     R / B, a short causal convolution per channel, and per token the projections' rows y' and x' (float32, biases included):
//       u   = conv_b + sum_j conv_w[c][taps-1-j] x'[t-j][c]           (zeros before the request's first token; no activation)
//       r   = sigmoid(Wa[b] u_b + ba),  i = sigmoid(Wi[b] u_b + bi)    per block b, Wa[b] and Wi[b] square
//       a   = exp(-c r softplus(lam)),  S <- a S + sqrt(1 - a^2) (i u)  c a constant of the design (an argument)
//       out = S * gelu_tanh(y')
//     State per slot: S [R], then the last taps - 1 rows x' [taps-1][R].
//     k_rglru_gates, a block per (tile of tokens, channel block): convolution into shared memory, then both gate products
//     with one output channel a thread (the matrices are given transposed, [b][in][out], so that a warp reads a row), then
//     a, the recurrence's input and the gated branch's activation.  k_rglru_scan, a thread a channel: the walk over a
//     portion's tokens, the read-out times the gated branch, and the slot's new tail.
//
// (2) Linear attention with a constant decay per head ("lightning attention"): S [D][V] per head,
//       S <- decay_h S + k v^T,   o = c S^T q,   q, k, v the projections' rows, behind an activation or as they are, c a constant.
//     k_decay_scan, a warp per eight value columns of a head: the state in registers, see there.
//     With a decay per key channel and token ("gated linear attention"), S <- diag(a_t) S + k v^T:
//       a_t = sigmoid(A2 (A1 h_t) + b)^(1/tau),   A1 h_t of a few values a token, columns of the same projection.
//     k_key_decay makes the rows a [n][H D]; the walk takes them beside q, k and v.
//
// (3) The state-space dual recurrence of Mamba-2: S [N][V] per head, head h reading key and query rows B, C of group h / (H / G),
//       S <- exp(-exp(A_log_h) dt) S + dt B x^T,   y = S^T C + D_h x,   dt = softplus(dt' + dt_bias_h)
//     with x, B, C behind a short causal convolution per channel (bias) and silu.  k_ssd_prep: the convolution and the two numbers
//     per token and head (decay, dt); the walk is k_decay_scan's with those in place of a constant decay.  State per slot:
//     S [H][V][N], then the last taps - 1 inputs of the convolution [taps-1][H V + 2 G N].
//
// Everything here is float32 in both precisions, and the walks go token by token: the state after a token does not depend
// on how the tokens were cut into steps, bit for bit.
#include "common.cuh"
#include "conv_tail.cuh"
#include <math.h>

#define RG_MAX_TAPS 16

// a weight through the read-only path (blocks of the same SM read the same rows), pinned where it is written like xr_ld_now
__device__ __forceinline__ float rc_ld_weight(const float* p) {
    float v;
    asm volatile("ld.global.nc.f32 %0, [%1];" : "=f"(v) : "l"(p) : "memory");
    return v;
}
__device__ __forceinline__ float rc_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float rc_softplus(float z) { return z > 30.0f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float rc_silu(float z) { return z < -80.0f ? 0.0f : z / (1.0f + expf(-z)); }
__device__ __forceinline__ float rc_gelu_tanh(float z) { return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))); }

#define RG_COLS 128              // output channels a block of the gates kernel takes (a thread each)

// The convolution of tokens t0 .. t0 + nt - 1 over the channels of block b into shared memory; u[e * stride_e + tt * stride_t].
__device__ __forceinline__ void rg_conv_tile(float* u, int stride_e, int stride_t, const float* __restrict__ proj, long long ldp, int x_col,
                                             const float* __restrict__ conv_w, const float* __restrict__ conv_b, const float* __restrict__ state,
                                             long long state_stride, const int* __restrict__ tok_seg, const int* __restrict__ seg_start,
                                             const int* __restrict__ seg_slot, int t0, int nt, int c0, int R, int Bs, int taps) {
    for (int idx = threadIdx.x; idx < nt * Bs; idx += blockDim.x) {
        const int tt = idx / Bs, e = idx % Bs, t = t0 + tt, ch = c0 + e;
        const int seg = tok_seg[t], i = t - seg_start[seg];
        const float* tail = state + (size_t)seg_slot[seg] * state_stride + R;
        const float* w = conv_w + (size_t)ch * taps;
        float acc = conv_b[ch];
        for (int j = taps - 1; j >= 0; j--) {                            // oldest input first
            const int ip = i - j;
            const float x = ip >= 0 ? proj[(size_t)(t - j) * ldp + x_col + ch] : tail[(size_t)(taps - 1 + ip) * R + ch];
            acc = fmaf(w[taps - 1 - j], x, acc);
        }
        u[e * stride_e + tt * stride_t] = acc;
    }
}

// a and the recurrence's input from the gates' sums; the gated branch's activation in place (nothing else reads those columns)
__device__ __forceinline__ void rg_finish(float ra, float ri, float u, float rate, float* a_out, float* b_out, float* y) {
    *y = rc_gelu_tanh(*y);
    const float log_a = rate * rc_sigmoid(ra);
    *a_out = expf(log_a);
    *b_out = sqrtf(-expm1f(2.0f * log_a)) * (rc_sigmoid(ri) * u);          // sqrt(1 - a^2) without the cancellation near a = 1
}

// Many tokens: a block per (TT tokens, channel block, 64 output channels), a thread an output channel with TT sums of each gate.
// The tile of u lies in shared memory input-major, [in][TT], so that a thread reads four tokens' values at once.
template <int TT>
__global__ void __launch_bounds__(RG_COLS)
k_rglru_gates(float* __restrict__ proj, long long ldp, int y_col, int x_col, const float* __restrict__ conv_w, const float* __restrict__ conv_b,
              const float* __restrict__ wa_t, const float* __restrict__ wi_t, const float* __restrict__ ba, const float* __restrict__ bi,
              const float* __restrict__ lam, const float* __restrict__ state, long long state_stride, const int* __restrict__ tok_seg,
              const int* __restrict__ seg_start, const int* __restrict__ seg_slot, float* __restrict__ a_out, float* __restrict__ b_out,
              int n, int R, int Bs, int taps, float c) {
    xr_pdl_launch();
    extern __shared__ __align__(16) float rg_u[];                // [Bs][TT]
    const int t0 = blockIdx.x * TT, b = blockIdx.y, c0 = b * Bs;
    const int nt = min(TT, n - t0);
    xr_pdl_wait();
    if (nt < TT)
        for (int idx = threadIdx.x; idx < TT * Bs; idx += blockDim.x) rg_u[idx] = 0.f;
    __syncthreads();
    rg_conv_tile(rg_u, TT, 1, (const float*)proj, ldp, x_col, conv_w, conv_b, state, state_stride, tok_seg, seg_start, seg_slot, t0, nt, c0, R, Bs, taps);
    __syncthreads();
    const float* wa = wa_t + (size_t)b * Bs * Bs;
    const float* wi = wi_t + (size_t)b * Bs * Bs;
    for (int o = blockIdx.z * RG_COLS + threadIdx.x; o < Bs; o += gridDim.z * RG_COLS) {
        float ra[TT], ri[TT];
#pragma unroll
        for (int tt = 0; tt < TT; tt++) { ra[tt] = ba[c0 + o]; ri[tt] = bi[c0 + o]; }
        // eight inputs' weights are fetched in one run of loads ahead of their multiply-adds (they come from the L2 cache, and
        // the few warps an SM holds of this kernel do not hide that latency otherwise)
        for (int k0 = 0; k0 < Bs; k0 += 8) {
            float va[8], vi[8];
#pragma unroll
            for (int kk = 0; kk < 8; kk++) {
                const int k = min(k0 + kk, Bs - 1);
                va[kk] = rc_ld_weight(wa + (size_t)k * Bs + o); vi[kk] = rc_ld_weight(wi + (size_t)k * Bs + o);
            }
#pragma unroll
            for (int kk = 0; kk < 8; kk++) { xr_ld_fence(va[kk]); xr_ld_fence(vi[kk]); }
#pragma unroll
            for (int kk = 0; kk < 8; kk++) {
                if (k0 + kk < Bs) {
                    const float4* uk = reinterpret_cast<const float4*>(rg_u + (size_t)(k0 + kk) * TT);
#pragma unroll
                    for (int q4 = 0; q4 < TT / 4; q4++) {
                        const float4 u = uk[q4];
                        ra[4 * q4] = fmaf(va[kk], u.x, ra[4 * q4]); ri[4 * q4] = fmaf(vi[kk], u.x, ri[4 * q4]);
                        ra[4 * q4 + 1] = fmaf(va[kk], u.y, ra[4 * q4 + 1]); ri[4 * q4 + 1] = fmaf(vi[kk], u.y, ri[4 * q4 + 1]);
                        ra[4 * q4 + 2] = fmaf(va[kk], u.z, ra[4 * q4 + 2]); ri[4 * q4 + 2] = fmaf(vi[kk], u.z, ri[4 * q4 + 2]);
                        ra[4 * q4 + 3] = fmaf(va[kk], u.w, ra[4 * q4 + 3]); ri[4 * q4 + 3] = fmaf(vi[kk], u.w, ri[4 * q4 + 3]);
                    }
                }
            }
        }
        const float rate = -c * rc_softplus(lam[c0 + o]);
#pragma unroll
        for (int tt = 0; tt < TT; tt++) {
            if (tt < nt) {
                const size_t at = (size_t)(t0 + tt) * R + c0 + o;
                rg_finish(ra[tt], ri[tt], rg_u[(size_t)o * TT + tt], rate, a_out + at, b_out + at, proj + (size_t)(t0 + tt) * ldp + y_col + c0 + o);
            }
        }
    }
}

// The convolution alone, a thread an element: u [n][R].  Ahead of k_rglru_gates_few, whose many small blocks would each compute
// the whole tile again behind a chain of dependent loads.
__global__ void k_rglru_conv(const float* __restrict__ proj, long long ldp, int x_col, const float* __restrict__ conv_w,
                             const float* __restrict__ conv_b, const float* __restrict__ state, long long state_stride,
                             const int* __restrict__ tok_seg, const int* __restrict__ seg_start, const int* __restrict__ seg_slot,
                             float* __restrict__ u, int n, int R, int taps) {
    xr_pdl_launch();
    const int idx = blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= n * R) return;
    const int t = idx / R, ch = idx % R;
    const int seg = tok_seg[t], i = t - seg_start[seg];
    const float* tail = state + (size_t)seg_slot[seg] * state_stride + R;
    const float* w = conv_w + (size_t)ch * taps;
    float acc = conv_b[ch];
    xr_pdl_wait();
    for (int j = taps - 1; j >= 0; j--) {                            // oldest input first
        const int ip = i - j;
        const float x = ip >= 0 ? proj[(size_t)(t - j) * ldp + x_col + ch] : tail[(size_t)(taps - 1 + ip) * R + ch];
        acc = fmaf(w[taps - 1 - j], x, acc);
    }
    u[idx] = acc;
}

// Few tokens (a step of single tokens): a warp an output channel, its lanes share the inputs, so that the matrices' rows (as
// stored, [b][out][in]) are read by whole warps and every load of a thread is in flight at once.  A block: 8 tokens, 8 channels.
__global__ void __launch_bounds__(256)
k_rglru_gates_few(float* __restrict__ proj, long long ldp, int y_col, int x_col, const float* __restrict__ conv_w, const float* __restrict__ conv_b,
                  const float* __restrict__ wa, const float* __restrict__ wi, const float* __restrict__ ba, const float* __restrict__ bi,
                  const float* __restrict__ lam, const float* __restrict__ state, long long state_stride, const int* __restrict__ tok_seg,
                  const int* __restrict__ seg_start, const int* __restrict__ seg_slot, float* __restrict__ a_out, float* __restrict__ b_out,
                  int n, int R, int Bs, int taps, float c, int groups, const float* __restrict__ u_in) {
    xr_pdl_launch();
    extern __shared__ __align__(16) float rg_u[];                // [8][Bs]
    const int t0 = blockIdx.x * 8, b = blockIdx.y / groups, c0 = b * Bs;
    const int nt = min(8, n - t0);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int o = (blockIdx.y % groups) * 8 + warp;
    xr_pdl_wait();
    for (int idx = threadIdx.x; idx < nt * Bs; idx += blockDim.x) rg_u[idx] = u_in[(size_t)(t0 + idx / Bs) * R + c0 + idx % Bs];
    __syncthreads();
    if (o >= Bs) return;
    const float* rowa = wa + ((size_t)b * Bs + o) * Bs;
    const float* rowi = wi + ((size_t)b * Bs + o) * Bs;
    float ra[8], ri[8];
#pragma unroll
    for (int tt = 0; tt < 8; tt++) { ra[tt] = 0.f; ri[tt] = 0.f; }
#pragma unroll 4
    for (int k = lane; k < Bs; k += 32) {
        const float va = rowa[k], vi = rowi[k];
#pragma unroll
        for (int tt = 0; tt < 8; tt++) {
            const float u = tt < nt ? rg_u[tt * Bs + k] : 0.f;
            ra[tt] = fmaf(va, u, ra[tt]);
            ri[tt] = fmaf(vi, u, ri[tt]);
        }
    }
#pragma unroll
    for (int tt = 0; tt < 8; tt++) { ra[tt] = xr_warp_sum(ra[tt]); ri[tt] = xr_warp_sum(ri[tt]); }
    const float rate = -c * rc_softplus(lam[c0 + o]);
#pragma unroll
    for (int tt = 0; tt < 8; tt++) {
        if (lane == tt && tt < nt) {
            const size_t at = (size_t)(t0 + tt) * R + c0 + o;
            rg_finish(ra[tt] + ba[c0 + o], ri[tt] + bi[c0 + o], rg_u[tt * Bs + o], rate, a_out + at, b_out + at, proj + (size_t)(t0 + tt) * ldp + y_col + c0 + o);
        }
    }
}

template <typename T>
__global__ void __launch_bounds__(128)
k_rglru_scan(const float* __restrict__ proj, long long ldp, int y_col, int x_col, const float* __restrict__ a_in, const float* __restrict__ b_in,
             float* __restrict__ state, long long state_stride, const int* __restrict__ seg_start, const int* __restrict__ seg_len,
             const int* __restrict__ seg_slot, T* __restrict__ out, int R, int taps) {
    xr_pdl_launch();
    const int ch = blockIdx.x * blockDim.x + threadIdx.x, seg = blockIdx.y;
    if (ch >= R) return;
    const int start = seg_start[seg], len = seg_len[seg];
    float* st = state + (size_t)seg_slot[seg] * state_stride;
    xr_pdl_wait();
    float S = st[ch];
    // The walk is a chain of dependent multiply-adds and nothing else hides the loads' latency: eight tokens' values are fetched in
    // one run of loads, and the next eight are on their way while these are walked.  (The gated branch's columns hold their
    // activation already: the gates kernel left it there.)
    float a[8], b[8], y[8], na[8], nb[8], ny[8];
    auto fetch = [&](int i0, float* fa, float* fb, float* fy) {
#pragma unroll
        for (int k = 0; k < 8; k++) {
            const size_t t = (size_t)(start + min(i0 + k, len - 1));
            fa[k] = xr_ld_now(a_in + t * R + ch); fb[k] = xr_ld_now(b_in + t * R + ch); fy[k] = xr_ld_now(proj + t * ldp + y_col + ch);
        }
#pragma unroll
        for (int k = 0; k < 8; k++) { xr_ld_fence(fa[k]); xr_ld_fence(fb[k]); xr_ld_fence(fy[k]); }
    };
    if (len > 0) fetch(0, na, nb, ny);
    for (int i0 = 0; i0 < len; i0 += 8) {
#pragma unroll
        for (int k = 0; k < 8; k++) { a[k] = na[k]; b[k] = nb[k]; y[k] = ny[k]; }
        if (i0 + 8 < len) fetch(i0 + 8, na, nb, ny);
#pragma unroll
        for (int k = 0; k < 8; k++) {
            if (i0 + k < len) {
                S = fmaf(a[k], S, b[k]);
                out[(size_t)(start + i0 + k) * R + ch] = xr_from_f32<T>(S * y[k]);
            }
        }
    }
    st[ch] = S;
    // the slot's tail becomes the last taps - 1 inputs of the convolution: rows of this portion, older ones from the tail as it was
    float keep[RG_MAX_TAPS];
    float* tail = st + R;
    for (int r = 0; r < taps - 1; r++) {
        const int i = len - (taps - 1) + r;
        keep[r] = i >= 0 ? proj[(size_t)(start + i) * ldp + x_col + ch] : tail[(size_t)(r + len) * R + ch];
    }
    for (int r = 0; r < taps - 1; r++) tail[(size_t)r * R + ch] = keep[r];
}

// proj [n][ldp] float32: the gated branch's pre-activations at y_col, the convolution's inputs at x_col, R columns each.
// conv_w [R][taps], conv_b [R]; wa_t, wi_t [B][R/B (in)][R/B (out)] and wa, wi the same matrices as stored, [B][out][in]; ba, bi,
// lam [R]; all float32.
// state [slots][state_stride] float32: S [R], tail [taps-1][R].  a_s, b_s, u_s [n][R] float32 scratch.  out [n][R] dtype `dtype`.
XR_EXPORT int xr_rglru(float* proj, long long ldp, int y_col, int x_col, const float* conv_w, const float* conv_b, const float* wa_t,
                       const float* wi_t, const float* wa, const float* wi, const float* ba, const float* bi, const float* lam, float* state, long long state_stride,
                       const int* tok_seg, const int* seg_start, const int* seg_len, const int* seg_slot, float* a_s, float* b_s, float* u_s, void* out,
                       int dtype, int n, int n_seg, int R, int B, int taps, float c, cudaStream_t stream) {
    if (n < 1 || n_seg < 1 || R < 1 || B < 1 || R % B || taps < 1 || taps > RG_MAX_TAPS || n_seg > 65535 || B > 65535 ||
        state_stride < (long long)R * taps)
        return XR_ERR_ARG;
    const int Bs = R / B;
    // (a tile of eight tokens of one channel block in shared memory: wide blocks ask for more than the default 48 KB)
    const size_t smem8 = (size_t)8 * Bs * sizeof(float);
    if (smem8 > 200 * 1024) return XR_ERR_ARG;
    if (smem8 > 48 * 1024 &&
        (cudaFuncSetAttribute(k_rglru_gates_few, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem8) != cudaSuccess ||
         cudaFuncSetAttribute(k_rglru_gates<8>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem8) != cudaSuccess))
        return XR_ERR_LAUNCH;
#define RG_ARGS(A, I) proj, ldp, y_col, x_col, conv_w, conv_b, A, I, ba, bi, lam, (const float*)state, state_stride, tok_seg, seg_start, seg_slot, a_s, b_s, n, R, Bs, taps, c
    if (n <= 16) {
        const int groups = (Bs + 7) / 8;
        xr_launch(k_rglru_conv, dim3((n * R + 255) / 256), dim3(256), 0, stream, (const float*)proj, ldp, x_col, conv_w, conv_b, (const float*)state,
                  state_stride, tok_seg, seg_start, seg_slot, u_s, n, R, taps);
        xr_launch(k_rglru_gates_few, dim3((n + 7) / 8, B * groups), dim3(256), smem8, stream, RG_ARGS(wa, wi), groups, (const float*)u_s);
    } else if (n >= 64 && (size_t)32 * Bs * sizeof(float) <= 48 * 1024) {
        xr_launch((k_rglru_gates<32>), dim3((n + 31) / 32, B, (Bs + RG_COLS - 1) / RG_COLS), dim3(RG_COLS), (size_t)32 * Bs * sizeof(float), stream, RG_ARGS(wa_t, wi_t));
    } else {
        xr_launch((k_rglru_gates<8>), dim3((n + 7) / 8, B, (Bs + RG_COLS - 1) / RG_COLS), dim3(RG_COLS), smem8, stream, RG_ARGS(wa_t, wi_t));
    }
#undef RG_ARGS
    dim3 gs((R + 127) / 128, n_seg);
    // (a step with long portions is a few long-lived blocks: they start behind the gates kernel, not into its last wave)
    const bool walk = n > 4 * n_seg;
    if (walk && dtype == XR_F32)
        xr_launch_behind((k_rglru_scan<float>), gs, dim3(128), 0, stream, (const float*)proj, ldp, y_col, x_col, (const float*)a_s, (const float*)b_s, state,
                         state_stride, seg_start, seg_len, seg_slot, (float*)out, R, taps);
    else if (walk && dtype == XR_BF16)
        xr_launch_behind((k_rglru_scan<__nv_bfloat16>), gs, dim3(128), 0, stream, (const float*)proj, ldp, y_col, x_col, (const float*)a_s, (const float*)b_s, state,
                         state_stride, seg_start, seg_len, seg_slot, (__nv_bfloat16*)out, R, taps);
    else if (dtype == XR_F32)
        xr_launch((k_rglru_scan<float>), gs, dim3(128), 0, stream, (const float*)proj, ldp, y_col, x_col, (const float*)a_s, (const float*)b_s, state,
                  state_stride, seg_start, seg_len, seg_slot, (float*)out, R, taps);
    else if (dtype == XR_BF16)
        xr_launch((k_rglru_scan<__nv_bfloat16>), gs, dim3(128), 0, stream, (const float*)proj, ldp, y_col, x_col, (const float*)a_s, (const float*)b_s, state,
                  state_stride, seg_start, seg_len, seg_slot, (__nv_bfloat16*)out, R, taps);
    else return XR_ERR_ARG;
    return xr_launch_status();
}

// ---------------------------------------------------------------------------------------------
// A block of eight warps owns VC * 8 value columns of one head, a warp VC of them; a warp's lanes share the key rows (lane l has rows l JD ..
// l JD + JD - 1), so a column's state lies in JD registers of every lane.  Per token a lane updates its JD x VC state elements
// and adds them, times q, into VC sums.  The sums of 32 / VC tokens are added over the lanes together: 32 numbers a lane, halved
// five times by an exchange with the lane 16, 8, 4, 2, 1 away, after which every lane holds one (token, column) sum and stores
// it: 31 shuffles for 32 / VC tokens, and one chain of five exchanges instead of one per token.
// Two elements are updated at a time by packed float32 multiply-adds (f32x2).  The tokens' q, k and v come in chunks of CH tokens
// through shared memory, two buffers: the next chunk's values are copied asynchronously while this chunk is walked (16 bytes a copy
// where sizes and addresses allow: VEC).  A step of many tokens applies silu to the rows beforehand, in place (k_silu_cols); a step
// of few applies it in shared memory.  A column's D state values lie together in memory ([H][V][D]), a lane's JD of them side by side.
// KIND: DS_HEAD: a constant decay per head.  DS_KEY: a decay per key channel and token, rows [n][H D] of their own.
// DS_SSD: the decay and the factor on the value come per token and head (coef), heads share key and query rows by `rep`, the
// value times skip[h] joins the read-out, and the blocks of a portion leave the convolution's new tail behind the walk.
#define DA_WARPS 8
#define DS_HEAD 0
#define DS_SSD 1
#define DS_KEY 2

struct SsdArgs {
    const float* coef;           // [n][H][2]: decay, dt
    const float* skip;           // [H]
    const float* raw;            // the convolution's inputs, row stride ld_raw, CH columns
    long long ld_raw;
    int CH, taps, rep;
};
struct KeyDecayArgs {
    const float* rows;           // [n][H D]: the decays
    float read_scale;            // factor on the read-outs (DS_HEAD too)
};

__global__ void k_silu_cols(float* __restrict__ rows, long long ld, int cols, size_t total) {
    xr_pdl_launch();
    xr_pdl_wait();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
        float* p = rows + (i / cols) * ld + (i % cols);
        *p = rc_silu(*p);
    }
}

// Two floats in one 64-bit register, and the packed arithmetic on them (each half rounded as the scalar operation is).
typedef unsigned long long F2;
__device__ __forceinline__ F2 f2_pack(float lo, float hi) { F2 r; asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi)); return r; }
__device__ __forceinline__ float2 f2_unpack(F2 v) { float2 r; asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v)); return r; }
__device__ __forceinline__ F2 f2_mul(F2 a, F2 b) { F2 r; asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b)); return r; }
__device__ __forceinline__ F2 f2_fma(F2 a, F2 b, F2 c) { F2 r; asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c)); return r; }

template <int BYTES>
__device__ __forceinline__ void rc_copy_async(float* dst, const float* src) {
    const unsigned at = (unsigned)__cvta_generic_to_shared(dst);
    if constexpr (BYTES == 16) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(at), "l"(src) : "memory");
    else asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(at), "l"(src) : "memory");
}
__device__ __forceinline__ void rc_copy_wait() { asm volatile("cp.async.wait_all;" ::: "memory"); }

// A lane's values of one token (JD of them) as pairs (JD 1: the value twice)
template <int JD>
__device__ __forceinline__ void rc_lane_values(const float* row, int lane, F2* out) {
    if constexpr (JD == 1) { const float x = row[lane]; out[0] = f2_pack(x, x); }
    else if constexpr (JD == 2) out[0] = *reinterpret_cast<const F2*>(row + 2 * lane);
    else {
#pragma unroll
        for (int j = 0; j < JD; j += 4) {
            const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(row + lane * JD + j);
            out[j / 2] = x.x; out[j / 2 + 1] = x.y;
        }
    }
}

// (blocks an SM: one where the walk's length counts, whose loads then have the registers to run ahead; two where there are many blocks)
template <int JD, int VC, int CH, bool VEC, int KIND>
__global__ void __launch_bounds__(32 * DA_WARPS, JD == 1 || (JD <= 4 && VC == 4) ? 2 : 1)
k_decay_scan(const float* __restrict__ proj, long long ldp, int q_col, int k_col, int v_col, const float* __restrict__ decay,
             float* __restrict__ state, long long state_stride, const int* __restrict__ seg_start, const int* __restrict__ seg_len,
             const int* __restrict__ seg_slot, float* __restrict__ o, int H, int D, int V, int activated, SsdArgs ssd, KeyDecayArgs key) {
    xr_pdl_launch();
    constexpr bool SSD = KIND == DS_SSD, KEY = KIND == DS_KEY;
    // a token's row in shared memory: q [DP], k [DP] (zeros behind D), DS_KEY: its decays [DP], the block's v [COLS]
    constexpr int COLS = VC * DA_WARPS, DP = 32 * JD, VA = (KEY ? 3 : 2) * DP, RW = VA + COLS, TB = 32 / VC, THREADS = 32 * DA_WARPS;
    // pairs: two neighbouring key channels of a lane (JD 1: two neighbouring value columns)
    constexpr int NP = JD == 1 ? 1 : JD / 2, NC = JD == 1 ? VC / 2 : VC;
    static_assert(CH % TB == 0 && VC % 2 == 0, "a chunk is whole batches of tokens");
    extern __shared__ __align__(16) float da_sm[];           // two chunks of CH rows
    __shared__ __align__(8) float da_coef[SSD ? 2 * CH * 2 : 2];       // SSD: a token's decay and dt
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int vb = blockIdx.x * COLS, v0 = vb + warp * VC, h = blockIdx.y, seg = blockIdx.z;
    const int start = seg_start[seg], len = seg_len[seg];
    const int g = SSD ? h / ssd.rep : h;                     // the head of the query and key rows
    const float dec = KIND == DS_HEAD ? decay[h] : 0.f, skip = SSD ? ssd.skip[h] : 0.f;
    float* slot = state + (size_t)seg_slot[seg] * state_stride;
    float* st = slot + (size_t)h * D * V;
    auto at = [&](int d, int c) -> size_t { return (size_t)(v0 + c) * D + d; };
    // (a chunk's columns behind D, and those of value columns that do not exist, are never copied to)
    if (D < DP || vb + COLS > V)
        for (int e = threadIdx.x; e < 2 * CH * RW; e += THREADS) da_sm[e] = 0.f;
    // ---- the copies of a chunk: 16 bytes each where sizes and addresses allow.  Where a thread's pieces lie is worked out once; a
    // chunk further they lie CH rows further.
    constexpr int UNIT = VEC ? 4 : 1, PIECES = CH * RW / UNIT, PER = (PIECES + THREADS - 1) / THREADS;
    auto source = [&](int e, long long& step) -> const float* {
        const int tok = e / RW, cc = e % RW;
        const float* row = proj + (size_t)(start + tok) * ldp;
        step = (long long)CH * ldp;
        if (e >= CH * RW) return nullptr;
        if (cc < DP) return cc < D ? row + q_col + g * D + cc : nullptr;
        if (cc < 2 * DP) return cc - DP < D ? row + k_col + g * D + cc - DP : nullptr;
        if (KEY && cc < VA) {
            step = (long long)CH * H * D;
            return cc - 2 * DP < D ? key.rows + ((size_t)(start + tok) * H + h) * D + cc - 2 * DP : nullptr;
        }
        return vb + cc - VA < V ? row + v_col + h * V + vb + cc - VA : nullptr;
    };
    const float* src[VEC ? PER : 1];
    long long step[VEC ? PER : 1];
    if constexpr (VEC) {
#pragma unroll
        for (int k = 0; k < PER; k++) src[k] = source(4 * (threadIdx.x + k * THREADS), step[k]);
    }
    auto load = [&](int chunk) {
        float* dst = da_sm + (chunk & 1) * CH * RW;
        if (SSD && threadIdx.x < 2 * CH) {
            const int i = chunk * CH + threadIdx.x / 2;
            if (i < len) rc_copy_async<4>(da_coef + (chunk & 1) * 2 * CH + threadIdx.x, ssd.coef + ((size_t)(start + i) * H + h) * 2 + (threadIdx.x & 1));
        }
        if constexpr (VEC) {
#pragma unroll
            for (int k = 0; k < PER; k++) {
                const int e = 4 * (threadIdx.x + k * THREADS);
                if (src[k] != nullptr) {
                    if (chunk * CH + e / RW < len) rc_copy_async<16>(dst + e, src[k]);
                    src[k] += step[k];
                }
            }
        } else {
            for (int e = threadIdx.x; e < CH * RW; e += THREADS) {
                long long st1;
                const float* p = chunk * CH + e / RW < len ? source(e, st1) : nullptr;
                if (p != nullptr) rc_copy_async<4>(dst + e, p + chunk * st1);
            }
        }
    };
    // behind the wait a thread may read what it copied itself: the activation in place
    auto arrive = [&](int chunk) {
        rc_copy_wait();
        if (!activated) {
            float* dst = da_sm + (chunk & 1) * CH * RW;
#pragma unroll 1
            for (int k = 0; k < PER; k++) {
                const int e = UNIT * (threadIdx.x + k * THREADS);
                if (e < CH * RW && chunk * CH + e / RW < len)
                    for (int i = 0; i < UNIT; i++) dst[e + i] = rc_silu(dst[e + i]);
            }
        }
    };
    xr_pdl_wait();
    const int chunks = (len + CH - 1) / CH;
    if (D < DP || vb + COLS > V) __syncthreads();            // (zeros stand before copies land beside them)
    if (chunks > 0) load(0);
    // ---- the state: a lane's JD elements of a column lie together: one access where they fall on a border of their size
    F2 s[NC][NP];
    const bool whole = JD > 1 && D % JD == 0 && ((uintptr_t)st % (JD >= 4 ? 16 : 8)) == 0;
    if constexpr (JD == 1) {
#pragma unroll
        for (int c = 0; c < NC; c++) {
            const bool a0 = lane < D && v0 + 2 * c < V, a1 = lane < D && v0 + 2 * c + 1 < V;
            s[c][0] = f2_pack(a0 ? st[at(lane, 2 * c)] : 0.f, a1 ? st[at(lane, 2 * c + 1)] : 0.f);
        }
    } else {
#pragma unroll
        for (int c = 0; c < VC; c++) {
            const bool ok = v0 + c < V;
            const float* p = st + at(lane * JD, ok ? c : 0);
#pragma unroll
            for (int j = 0; j < JD; j += 2) {
                const int d = lane * JD + j;
                if (whole && JD % 4 == 0) {
                    if (j % 4 == 0) {
                        const float4 x = ok && d < D ? *reinterpret_cast<const float4*>(p + j) : make_float4(0.f, 0.f, 0.f, 0.f);
                        s[c][j / 2] = f2_pack(x.x, x.y);
                        if (j / 2 + 1 < NP) s[c][j / 2 + 1] = f2_pack(x.z, x.w);
                    }
                } else if (whole) {
                    const float2 x = ok && d < D ? *reinterpret_cast<const float2*>(p + j) : make_float2(0.f, 0.f);
                    s[c][j / 2] = f2_pack(x.x, x.y);
                } else {
                    s[c][j / 2] = f2_pack(ok && d < D ? p[j] : 0.f, ok && d + 1 < D ? p[j + 1] : 0.f);
                }
            }
        }
    }
    if (chunks > 0) arrive(0);
    __syncthreads();
    for (int ch = 0; ch < chunks; ch++) {
        if (ch + 1 < chunks) load(ch + 1);
        const float* base = da_sm + (ch & 1) * CH * RW;
        const int here = min(CH, len - ch * CH);
#pragma unroll 1
        for (int t0 = 0; t0 < here; t0 += TB) {
            float acc[TB * VC];
#pragma unroll
            for (int k = 0; k < TB * VC; k++) acc[k] = 0.f;
            auto token = [&](int tb) {
                const float* row = base + (t0 + tb) * RW;
                F2 q[NP], k[NP], ak[KEY ? NP : 1], v[NC];
                rc_lane_values<JD>(row, lane, q);
                rc_lane_values<JD>(row + DP, lane, k);
                if constexpr (KEY) rc_lane_values<JD>(row + 2 * DP, lane, ak);
                float2 ad = make_float2(dec, 1.f);
                if constexpr (SSD) ad = *reinterpret_cast<const float2*>(da_coef + ((ch & 1) * CH + t0 + tb) * 2);
                const F2 a = f2_pack(ad.x, ad.x);
                float vf[VC];
                if constexpr (VC % 4 == 0) {
#pragma unroll
                    for (int c = 0; c < VC; c += 4) {
                        const float4 x = *reinterpret_cast<const float4*>(row + VA + warp * VC + c);
                        vf[c] = x.x; vf[c + 1] = x.y; vf[c + 2] = x.z; vf[c + 3] = x.w;
                    }
                } else {
#pragma unroll
                    for (int c = 0; c < VC; c += 2) {
                        const float2 x = *reinterpret_cast<const float2*>(row + VA + warp * VC + c);
                        vf[c] = x.x; vf[c + 1] = x.y;
                    }
                }
                if constexpr (SSD) {
#pragma unroll
                    for (int c = 0; c < VC; c++) vf[c] *= ad.y;
                }
#pragma unroll
                for (int c = 0; c < NC; c++) v[c] = JD == 1 ? f2_pack(vf[2 * c], vf[2 * c + 1]) : f2_pack(vf[c], vf[c]);
#pragma unroll
                for (int c = 0; c < NC; c++) {
                    F2 y;
#pragma unroll
                    for (int j = 0; j < NP; j++) {
                        s[c][j] = f2_fma(KEY ? ak[KEY ? j : 0] : a, s[c][j], f2_mul(k[j], v[c]));
                        y = j == 0 ? f2_mul(s[c][j], q[j]) : f2_fma(s[c][j], q[j], y);
                    }
                    const float2 sum = f2_unpack(y);
                    if constexpr (JD == 1) { acc[tb * VC + 2 * c] = sum.x; acc[tb * VC + 2 * c + 1] = sum.y; }
                    else acc[tb * VC + c] = sum.x + sum.y;
                }
            };
            // (a whole batch of tokens without a branch between them: their reads of shared memory are then in flight together)
            if (t0 + TB <= here) {
#pragma unroll
                for (int tb = 0; tb < TB; tb++) token(tb);
            } else {
#pragma unroll
                for (int tb = 0; tb < TB; tb++)
                    if (t0 + tb < here) token(tb);
            }
            // 32 sums a lane -> one: a lane whose bit is set keeps the upper half of what it carries and hands over the lower one
#pragma unroll
            for (int w = 16, bit = 16; w > 0; w >>= 1, bit >>= 1) {
                const bool upper = lane & bit;
#pragma unroll
                for (int c = 0; c < w; c++) {
                    const float send = upper ? acc[c] : acc[c + w], keep = upper ? acc[c + w] : acc[c];
                    acc[c] = keep + __shfl_xor_sync(0xffffffffu, send, bit);
                }
            }
            // the sum this lane holds: bit 16 of the lane chose the upper 16 of 32, bit 8 the upper 8 of those, ...: the lane's number
            // read from its highest bit down is the sum's index
            const int tb = lane / VC, c = lane % VC;
            if (t0 + tb < here && v0 + c < V) {
                float y = acc[0];
                if constexpr (SSD) y = fmaf(skip, base[(t0 + tb) * RW + VA + warp * VC + c], y);
                else y *= key.read_scale;
                o[(size_t)(start + ch * CH + t0 + tb) * H * V + (size_t)h * V + v0 + c] = y;
            }
        }
        if (ch + 1 < chunks) arrive(ch + 1);
        __syncthreads();
    }
    if constexpr (JD == 1) {
#pragma unroll
        for (int c = 0; c < NC; c++) {
            const float2 x = f2_unpack(s[c][0]);
            if (lane < D && v0 + 2 * c < V) st[at(lane, 2 * c)] = x.x;
            if (lane < D && v0 + 2 * c + 1 < V) st[at(lane, 2 * c + 1)] = x.y;
        }
    } else {
#pragma unroll
        for (int c = 0; c < VC; c++) {
            if (v0 + c >= V) continue;
            float* p = st + at(lane * JD, c);
#pragma unroll
            for (int j = 0; j < JD; j += 2) {
                const int d = lane * JD + j;
                const float2 x = f2_unpack(s[c][j / 2]);
                if (whole && JD % 4 == 0) {
                    if (j % 4 == 0 && d < D) {
                        const float2 y = f2_unpack(s[c][j / 2 + 1 < NP ? j / 2 + 1 : 0]);
                        *reinterpret_cast<float4*>(p + j) = make_float4(x.x, x.y, y.x, y.y);
                    }
                } else if (whole) {
                    if (d < D) *reinterpret_cast<float2*>(p + j) = x;
                } else {
                    if (d < D) p[j] = x.x;
                    if (d + 1 < D) p[j + 1] = x.y;
                }
            }
        }
    }
    if constexpr (SSD)
        if (ssd.taps > 1)
            xr_tail_update<float>(ssd.raw, ssd.ld_raw, slot + (size_t)H * V * D, start, len, ssd.CH, ssd.taps,
                                  blockIdx.y * gridDim.x + blockIdx.x, gridDim.x * gridDim.y);
}

// Value columns a warp: two where the walk's length is what counts (few blocks, each with its SM to itself), four where there are more
// blocks than the machine holds at once (half the reads of shared memory per state element).  A column's arithmetic is the same.
static inline bool decay_scan_wide(int V, int H, int n_seg) { return (long long)((V + 15) / 16) * H * n_seg > 2LL * xr_sm_count(); }

// bytes of shared memory a block of the walk takes: two chunks of CH tokens' rows
static constexpr size_t decay_scan_smem(int JD, int VC, int CH, int KIND) {
    return (size_t)2 * CH * ((KIND == DS_KEY ? 3 : 2) * 32 * JD + VC * DA_WARPS) * sizeof(float);
}

template <int KIND>
static int launch_decay_scan(const float* proj, long long ldp, int q_col, int k_col, int v_col, const float* decay, float* state, long long state_stride,
                             const int* seg_start, const int* seg_len, const int* seg_slot, float* o, int n, int n_seg, int H, int D, int V, bool ready,
                             KeyDecayArgs key, cudaStream_t stream) {
    // (a step with long portions is a few long-lived blocks: they start behind the kernel ahead, not into its last wave)
    const bool walk = n > 4 * n_seg;
    // 16 bytes a load where every row, column offset and size falls on a 16-byte border
    const bool vec = !((D | V | ldp | q_col | k_col | v_col) & 3) && !(((uintptr_t)proj | (uintptr_t)key.rows) & 15);
#define DS_ARGS(JD, VC, CH) dim3((V + VC * DA_WARPS - 1) / (VC * DA_WARPS), H, n_seg), dim3(32 * DA_WARPS), decay_scan_smem(JD, VC, CH, KIND), stream, \
                            proj, ldp, q_col, k_col, v_col, decay, state, state_stride, seg_start, seg_len, seg_slot, o, H, D, V, ready ? 1 : 0, SsdArgs{}, key
#define DS1(JD, VC, CH, VEC)                                                                                                                 \
    do {                                                                                                                                     \
        if (decay_scan_smem(JD, VC, CH, KIND) > 48 * 1024 &&                                                                                 \
            cudaFuncSetAttribute(k_decay_scan<JD, VC, CH, VEC, KIND>, cudaFuncAttributeMaxDynamicSharedMemorySize,                           \
                                 (int)decay_scan_smem(JD, VC, CH, KIND)) != cudaSuccess)                                                     \
            return XR_ERR_LAUNCH;                                                                                                            \
        if (walk) xr_launch_behind((k_decay_scan<JD, VC, CH, VEC, KIND>), DS_ARGS(JD, VC, CH));                                              \
        else xr_launch((k_decay_scan<JD, VC, CH, VEC, KIND>), DS_ARGS(JD, VC, CH));                                                          \
    } while (0)
#define DS(JD, VC, CH)                                                                                                                       \
    do {                                                                                                                                     \
        if (vec) DS1(JD, VC, CH, true);                                                                                                      \
        else DS1(JD, VC, CH, false);                                                                                                         \
    } while (0)
    const bool wide = decay_scan_wide(V, H, n_seg);
    if (D <= 32) DS(1, 2, 16);
    else if (D <= 64 && !wide) DS(2, 2, 16);
    else if (D <= 64) DS(2, 4, 16);
    else if (D <= 128 && !wide) DS(4, 2, 16);
    else if (D <= 128) DS(4, 4, 16);
    else DS(8, 4, 8);
#undef DS
#undef DS1
#undef DS_ARGS
    return xr_launch_status();
}

// proj [n][ldp] float32: q at q_col [H][D], k at k_col [H][D], v at v_col [H][V]; with `silu` their pre-activations (columns from the
// first of q to the last of v, which a step of many tokens activates in place), else as they are; decay [H] float32; state
// [slots][state_stride] float32, S [H][V][D];  o [n][H V] float32 receives the read-outs, times read_scale.
XR_EXPORT int xr_decay_attention(float* proj, long long ldp, int q_col, int k_col, int v_col, const float* decay, float* state,
                                 long long state_stride, const int* seg_start, const int* seg_len, const int* seg_slot, float* o, int n, int n_seg,
                                 int H, int D, int V, int silu, float read_scale, cudaStream_t stream) {
    if (n < 1 || n_seg < 1 || H < 1 || D < 1 || V < 1 || D > 256 || n_seg > 65535 || H > 65535 || state_stride < (long long)H * D * V)
        return XR_ERR_ARG;
    // q, k, v lie side by side from q_col on (the caller's layout): one pass activates them all
    const bool many = silu && n > 16 && k_col == q_col + H * D && v_col == k_col + H * D;
    if (many) {
        const size_t total = (size_t)n * (2 * H * D + H * V);
        const int blocks = (int)((total + 255) / 256 < (size_t)xr_sm_count() * 16 ? (total + 255) / 256 : xr_sm_count() * 16);
        xr_launch(k_silu_cols, dim3(blocks), dim3(256), 0, stream, proj + q_col, ldp, 2 * H * D + H * V, total);
    }
    return launch_decay_scan<DS_HEAD>(proj, ldp, q_col, k_col, v_col, decay, state, state_stride, seg_start, seg_len, seg_slot, o, n, n_seg, H, D, V,
                                      many || !silu, KeyDecayArgs{nullptr, read_scale}, stream);
}

// ---------------------------------------------------------------------------------------------
// Decays per key channel: out[t][c] = sigmoid(z)^(1/tau) = exp(log sigmoid(z) / tau), z = bias[c] + sum_r w_t[r][c] in[t][r]; `in` R
// columns of a wider float32 row, w_t the matrix transposed ([R][C], so that a warp reads a row).  A thread a channel with KD_T
// tokens' sums; the tokens' rows lie in shared memory, R of them at a time.
// ---------------------------------------------------------------------------------------------
#define KD_R 64
template <int KD_T>
__global__ void __launch_bounds__(128)
k_key_decay(const float* __restrict__ in, long long ld_in, const float* __restrict__ w_t, const float* __restrict__ bias, float* __restrict__ out,
            int n, int R, int C, float inv_tau, int early) {
    if (early) xr_pdl_launch();                  // (a walk of long portions stays behind this kernel: see xr_launch_behind)
    __shared__ float rows[KD_R][KD_T];
    const int c = blockIdx.x * 128 + threadIdx.x, t0 = blockIdx.y * KD_T, cc = min(c, C - 1);
    float z[KD_T];
    const float b = bias[cc];
#pragma unroll
    for (int i = 0; i < KD_T; i++) z[i] = b;
    xr_pdl_wait();
    for (int r0 = 0; r0 < R; r0 += KD_R) {
        const int rn = min(KD_R, R - r0);
        for (int e = threadIdx.x; e < rn * KD_T; e += 128) {
            const int t = t0 + e / rn, r = e % rn;
            rows[r][e / rn] = t < n ? in[(size_t)t * ld_in + r0 + r] : 0.f;
        }
        __syncthreads();
#pragma unroll 8
        for (int r = 0; r < rn; r++) {
            const float w = w_t[(size_t)(r0 + r) * C + cc];
#pragma unroll
            for (int i = 0; i < KD_T; i++) z[i] = fmaf(w, rows[r][i], z[i]);
        }
        __syncthreads();
    }
    if (c >= C) return;
#pragma unroll
    for (int i = 0; i < KD_T; i++)
        if (t0 + i < n) out[(size_t)(t0 + i) * C + c] = expf((fminf(z[i], 0.f) - log1pf(expf(-fabsf(z[i])))) * inv_tau);
}

// Linear attention with a decay per key channel: q, k, v as in xr_decay_attention without an activation; the decays' inner values at
// a_col (R columns of proj), w_t [R][H D], bias [H D] float32; decays [n][H D] float32 scratch.
XR_EXPORT int xr_key_decay_attention(const float* proj, long long ldp, int q_col, int k_col, int v_col, int a_col, const float* w_t, const float* bias,
                                     int R, float tau, float* decays, float* state, long long state_stride, const int* seg_start, const int* seg_len,
                                     const int* seg_slot, float* o, int n, int n_seg, int H, int D, int V, float read_scale, cudaStream_t stream) {
    if (n < 1 || n_seg < 1 || H < 1 || D < 1 || V < 1 || D > 256 || R < 1 || !(tau > 0.f) || n_seg > 65535 || H > 65535 || n > 65535 * 4 ||
        state_stride < (long long)H * D * V)
        return XR_ERR_ARG;
    const int C = H * D, early = n > 4 * n_seg ? 0 : 1;
    if (n > 64) xr_launch((k_key_decay<16>), dim3((C + 127) / 128, (n + 15) / 16), dim3(128), 0, stream, proj + a_col, ldp, w_t, bias, decays, n, R, C, 1.0f / tau, early);
    else xr_launch((k_key_decay<4>), dim3((C + 127) / 128, (n + 3) / 4), dim3(128), 0, stream, proj + a_col, ldp, w_t, bias, decays, n, R, C, 1.0f / tau, early);
    return launch_decay_scan<DS_KEY>(proj, ldp, q_col, k_col, v_col, nullptr, state, state_stride, seg_start, seg_len, seg_slot, o, n, n_seg, H, D, V,
                                     true, KeyDecayArgs{decays, read_scale}, stream);
}

// ---------------------------------------------------------------------------------------------
// (3): the convolution with its bias and silu, xbc [n][CH], and per token and head coef [n][H][2] = (exp(neg_a dt), dt), dt =
// softplus(dt' + dt_bias).  A thread a column of xbc or a head's dt, TT tokens one after the other.  TAPS: taps known at
// compile time (0: any number).
// ---------------------------------------------------------------------------------------------
template <int TAPS>
__global__ void __launch_bounds__(256)
k_ssd_prep(const float* __restrict__ proj, long long ldp, int x_col, int dt_col, const float* __restrict__ conv_w, const float* __restrict__ conv_b,
           const float* __restrict__ dt_bias, const float* __restrict__ neg_a, const float* __restrict__ state, long long state_stride,
           long long tail_off, const int* __restrict__ tok_seg, const int* __restrict__ seg_start, const int* __restrict__ seg_slot,
           float* __restrict__ xbc, float* __restrict__ coef, int n, int CH, int H, int taps, int TT, int early) {
    if (early) xr_pdl_launch();                  // (the walk behind it is a few long-lived blocks: see k_delta_prep)
    const int c = blockIdx.x * blockDim.x + threadIdx.x, t0 = blockIdx.y * TT, t1 = min(n, t0 + TT);
    if (c >= CH + H) return;
    if (c >= CH) {
        const int h = c - CH;
        const float bias = dt_bias[h], na = neg_a[h];
        xr_pdl_wait();
        for (int t = t0; t < t1; t++) {
            const float z = proj[(size_t)t * ldp + dt_col + h] + bias;
            const float dt = fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
            *reinterpret_cast<float2*>(coef + ((size_t)t * H + h) * 2) = make_float2(expf(na * dt), dt);
        }
        return;
    }
    const int K = TAPS > 0 ? TAPS : taps;
    const float* wc = conv_w + (size_t)c * K;
    const float bias = conv_b[c];
    float w[TAPS > 0 ? TAPS : 1];
    if constexpr (TAPS > 0) {
#pragma unroll
        for (int j = 0; j < TAPS; j++) w[j] = wc[j];
    }
    xr_pdl_wait();
    for (int t = t0; t < t1; t++) {
        const int seg = tok_seg[t], i = t - seg_start[seg];
        const float* x = proj + (size_t)t * ldp + x_col + c;
        float acc = bias;
        if (TAPS > 0 && i >= TAPS - 1) {                                   // every input is a row of this step
            float v[TAPS > 0 ? TAPS : 1];
#pragma unroll
            for (int j = 0; j < TAPS; j++) v[j] = x[-(long long)(TAPS - 1 - j) * ldp];
#pragma unroll
            for (int j = 0; j < TAPS; j++) acc = fmaf(w[j], v[j], acc);
        } else {
            const float* tail = state + (size_t)seg_slot[seg] * state_stride + tail_off;
            for (int j = K - 1; j >= 0; j--) {                             // oldest input first
                const int ip = i - j;
                const float v = ip >= 0 ? x[-(long long)j * ldp] : tail[(size_t)(K - 1 + ip) * CH + c];
                acc = fmaf(wc[K - 1 - j], v, acc);
            }
        }
        xbc[(size_t)t * CH + c] = rc_silu(acc);
    }
}

// proj [n][ldp] float32: the convolution's inputs x [H][V], B [G][N], C [G][N] from x_col on, dt' [H] at dt_col.  conv_w [CH][taps]
// (the last column the current token's), conv_b [CH], dt_bias, neg_a = -exp(A_log), skip [H]; all float32.
// state [slots][state_stride] float32.  xbc [n][CH], coef [n][H][2] float32 scratch.  y [n][H V] float32: S^T C + D x.
XR_EXPORT int xr_ssd(const float* proj, long long ldp, int x_col, int dt_col, const float* conv_w, const float* conv_b, const float* dt_bias,
                     const float* neg_a, const float* skip, float* state, long long state_stride, const int* tok_seg, const int* seg_start,
                     const int* seg_len, const int* seg_slot, float* xbc, float* coef, float* y, int n, int n_seg, int H, int G, int N, int V,
                     int taps, cudaStream_t stream) {
    if (n < 1 || n_seg < 1 || H < 1 || G < 1 || H % G || N < 1 || N > 256 || V < 1 || taps < 1 || taps > 64 || n_seg > 65535 || H > 65535)
        return XR_ERR_ARG;
    const int CH = H * V + 2 * G * N;
    const long long tail_off = (long long)H * V * N;
    if (state_stride < tail_off + (long long)(taps - 1) * CH) return XR_ERR_ARG;
    const int TT = n > 64 ? 8 : 1, early = n <= 64 ? 1 : 0;
    const dim3 gp((CH + H + 255) / 256, (n + TT - 1) / TT);
    if (gp.y > 65535) return XR_ERR_ARG;
#define SP(TAPS) xr_launch((k_ssd_prep<TAPS>), gp, dim3(256), 0, stream, proj, ldp, x_col, dt_col, conv_w, conv_b, dt_bias, neg_a, (const float*)state,      \
                           state_stride, tail_off, tok_seg, seg_start, seg_slot, xbc, coef, n, CH, H, taps, TT, early)
    if (taps == 4) SP(4);
    else SP(0);
#undef SP
    const bool walk = n > 4 * n_seg;
    const bool vec = !((N | V) & 3) && !((uintptr_t)xbc & 15);
    const SsdArgs ssd{coef, skip, proj + x_col, ldp, CH, taps, H / G};
#define SS_ARGS(JD, VC, CK) dim3((V + VC * DA_WARPS - 1) / (VC * DA_WARPS), H, n_seg), dim3(32 * DA_WARPS), decay_scan_smem(JD, VC, CK, DS_SSD), stream, (const float*)xbc, (long long)CH,            \
                    H * V + G * N, H * V, 0, (const float*)nullptr, state, state_stride, seg_start, seg_len, seg_slot, y, H, N, V, 1, ssd, KeyDecayArgs{nullptr, 1.0f}
#define SS1(JD, VC, CK, VEC)                                                                                                                 \
    do {                                                                                                                                     \
        if (walk) xr_launch_behind((k_decay_scan<JD, VC, CK, VEC, DS_SSD>), SS_ARGS(JD, VC, CK));                                                      \
        else xr_launch((k_decay_scan<JD, VC, CK, VEC, DS_SSD>), SS_ARGS(JD, VC, CK));                                                                  \
    } while (0)
#define SS(JD, VC, CK)                                                                                                                       \
    do {                                                                                                                                     \
        if (vec) SS1(JD, VC, CK, true);                                                                                                      \
        else SS1(JD, VC, CK, false);                                                                                                         \
    } while (0)
    const bool wide = decay_scan_wide(V, H, n_seg);
    if (N <= 32) SS(1, 2, 16);
    else if (N <= 64 && !wide) SS(2, 2, 16);
    else if (N <= 64) SS(2, 4, 16);
    else if (N <= 128 && !wide) SS(4, 2, 16);
    else if (N <= 128) SS(4, 4, 16);
    else SS(8, 4, 8);
#undef SS
#undef SS1
#undef SS_ARGS
    return xr_launch_status();
}
