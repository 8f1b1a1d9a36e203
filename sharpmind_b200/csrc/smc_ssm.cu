// State-space (Mamba-2) sequence mixing between its two projections:
//   x | B | C pass a causal convolution per channel and SiLU;  dt = softplus(dt_raw + bias)
//   S_t = exp(-exp(A_log) dt) S_{t-1} + dt B_t x_t^T,   y_t = S_t^T C_t + D x_t        per head, S [state, vdim]
//   o = RMSNorm in parts(y * SiLU(z)) * w
// dt, decays, S and y are fp32.  A sequence's state is S and the inputs of the convolution's last taps (position p in row
// p % taps of its ring).
#include <cuda_bf16.h>

#include "smc_common.cuh"

namespace {

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16_rn(v); }
__device__ __forceinline__ float silu(float z) { return __fdiv_rn(z, 1.0f + expf(-z)); }
__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// ------------------------------------------------------------------------------ convolution
// A thread per channel walks CR rows.  Inputs before the portion come from the ring; those before position 0 are zero.
// One row per sequence (decoding): the same launch stores the row's input, whose ring place nobody reads any more.
constexpr int CR = 8;
template <typename T>
__global__ void __launch_bounds__(128) ssm_conv_kernel(const T *__restrict__ zx, int ld, int inner, T *__restrict__ out, T *__restrict__ ring, smc_rows rw,
                                                       const float *__restrict__ w, const float *__restrict__ b, int ch, int taps)
{
    smc_grid_dep_sync();
    const int c = blockIdx.x * 128 + threadIdx.x;
    if (c >= ch) return;
    const int r0 = blockIdx.y * (rw.seq0 >= 0 ? CR : 1), r1 = min(rw.n, r0 + (rw.seq0 >= 0 ? CR : 1));
    const int slot = rw.seq0 >= 0 ? rw.seq0 : r0, p0 = rw.pos[slot] - (rw.seq0 >= 0 ? 0 : r0);  // row r is at position p0 + r
    T *rg = ring + (size_t)slot * taps * ch + c;
    const float *wc = w + (size_t)c * taps;
    const float bias = b[c];
    for (int r = r0; r < r1; ++r) {
        const int p = p0 + r, first = rw.seq0 >= 0 ? 0 : r;  // rows before `first` belong to other sequences
        float acc = bias;
        for (int j = taps - 1; j >= 0; --j) {  // oldest first
            if (p - j < 0) continue;
            const T v = r - j >= first ? zx[(size_t)(r - j) * ld + inner + c] : rg[(size_t)((p - j) % taps) * ch];
            acc = fmaf(wc[taps - 1 - j], to_f(v), acc);
        }
        out[(size_t)r * ch + c] = from_f<T>(silu(acc));
        if (rw.seq0 < 0 || rw.n == 1) rg[(size_t)(p % taps) * ch] = zx[(size_t)r * ld + inner + c];
    }
}

// The last `taps` inputs of a portion of several rows, after every reader of the old ones is done.
template <typename T>
__global__ void __launch_bounds__(128) ssm_conv_keep_kernel(const T *__restrict__ zx, int ld, int inner, T *__restrict__ ring, smc_rows rw, int ch,
                                                            int taps)
{
    smc_grid_dep_sync();
    const int c = blockIdx.x * 128 + threadIdx.x, r = rw.n - 1 - (int)blockIdx.y;
    if (c >= ch || r < 0) return;
    const int p = rw.pos[rw.seq0] + r;
    ring[((size_t)rw.seq0 * taps + p % taps) * ch + c] = zx[(size_t)r * ld + inner + c];
}

// ------------------------------------------------------------------------------ recurrence, token after token
// A CTA: one head of one sequence, 16 value columns; eight lanes share a column, lane i holding states i, i + 8, ....
// Steps are staged sixteen at a time.
constexpr int SC = 16;
template <typename T, int NPL>
__global__ void __launch_bounds__(128) ssm_scan_kernel(const T *__restrict__ xbc, const float *__restrict__ dt_raw, float *__restrict__ y,
                                                       float *__restrict__ state, smc_rows rw, const float *__restrict__ dt_bias,
                                                       const float *__restrict__ a_log, const float *__restrict__ d_skip, int heads, int P, int N,
                                                       int groups)
{
    extern __shared__ float sm[];
    float *sB = sm, *sC = sB + SC * N, *sx = sC + SC * N, *sdt = sx + SC * 16, *sa = sdt + SC;
    smc_grid_dep_sync();
    const int h = blockIdx.x, c0 = blockIdx.y * 16, sub = threadIdx.x & 7, col = threadIdx.x >> 3, p = c0 + col;
    const int slot = rw.seq0 >= 0 ? rw.seq0 : (int)blockIdx.z, row0 = rw.seq0 >= 0 ? 0 : (int)blockIdx.z, T_ = rw.seq0 >= 0 ? rw.n : 1;
    const bool fresh = rw.pos[slot] == 0;
    const int inner = heads * P, ch = inner + 2 * groups * N, g = h / (heads / groups);
    float *st = state + (((size_t)slot * heads + h) * P + min(p, P - 1)) * N;
    float S[NPL];
#pragma unroll
    for (int j = 0; j < NPL; ++j) {
        const int n = sub + 8 * j;
        S[j] = !fresh && n < N ? st[n] : 0.f;
    }
    const float A = -expf(a_log[h]), D = d_skip[h], bias = dt_bias[h];
    for (int t0 = 0; t0 < T_; t0 += SC) {
        const int nt = min(SC, T_ - t0);
        __syncthreads();
        for (int e = threadIdx.x; e < nt * N; e += 128) {
            const T *src = xbc + (size_t)(row0 + t0 + e / N) * ch + inner + g * N + e % N;
            sB[e] = to_f(src[0]), sC[e] = to_f(src[groups * N]);
        }
        for (int e = threadIdx.x; e < nt * 16; e += 128)
            sx[e] = c0 + (e & 15) < P ? to_f(xbc[(size_t)(row0 + t0 + (e >> 4)) * ch + h * P + c0 + (e & 15)]) : 0.f;
        if (threadIdx.x < nt) {
            const float dt = softplus(dt_raw[(size_t)(row0 + t0 + threadIdx.x) * heads + h] + bias);
            sdt[threadIdx.x] = dt, sa[threadIdx.x] = expf(A * dt);
        }
        __syncthreads();
        for (int t = 0; t < nt; ++t) {
            const float a = sa[t], x = sx[t * 16 + col], dx = sdt[t] * x;
            float acc = 0.f;
#pragma unroll
            for (int j = 0; j < NPL; ++j) {
                const int n = sub + 8 * j;
                if (n < N) {
                    S[j] = fmaf(sB[t * N + n], dx, a * S[j]);
                    acc = fmaf(S[j], sC[t * N + n], acc);
                }
            }
            acc += __shfl_xor_sync(0xffffffffu, acc, 1);
            acc += __shfl_xor_sync(0xffffffffu, acc, 2);
            acc += __shfl_xor_sync(0xffffffffu, acc, 4);
            if (sub == 0 && p < P) y[(size_t)(row0 + t0 + t) * inner + h * P + p] = fmaf(D, x, acc);
        }
    }
    if (p < P) {
#pragma unroll
        for (int j = 0; j < NPL; ++j)
            if (sub + 8 * j < N) st[sub + 8 * j] = S[j];
    }
}

// ------------------------------------------------------------------------------ gate, then norm in parts
template <typename T>
__global__ void __launch_bounds__(128) ssm_gate_norm_kernel(const float *__restrict__ y, const T *__restrict__ zx, int ld, const float *__restrict__ w,
                                                            T *__restrict__ o, int inner, int parts, float eps)
{
    extern __shared__ float sv[];
    __shared__ float red[4];
    smc_grid_dep_sync();
    const int n = inner / parts, r = blockIdx.x, base = blockIdx.y * n;
    float ss = 0.f;
    for (int i = threadIdx.x; i < n; i += 128) {
        const float v = y[(size_t)r * inner + base + i] * silu(to_f(zx[(size_t)r * ld + base + i]));
        sv[i] = v;
        ss = fmaf(v, v, ss);
    }
    ss = smc_group_sum<32>(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = (red[0] + red[1]) + (red[2] + red[3]);
    const float inv = __fdiv_rn(1.0f, sqrtf(__fdiv_rn(ss, (float)n) + eps));
    for (int i = threadIdx.x; i < n; i += 128) o[(size_t)r * inner + base + i] = from_f<T>((sv[i] * inv) * w[base + i]);
}

template <typename T>
int mix(smc_ctx *ctx, const smc_ssm_dims &d, const smc_ssm_bufs &b, const smc_rows &rw, const float *conv_w, const float *conv_b, const float *dt_bias,
        const float *a_log, const float *d_skip, const float *norm, cudaStream_t s)
{
    const int inner = d.heads * d.vdim, ch = inner + 2 * d.groups * d.state;
    const bool seq = rw.seq0 >= 0;
    smc_launch_dep(ctx->use_pdl, ssm_conv_kernel<T>, dim3((ch + 127) / 128, seq ? (rw.n + CR - 1) / CR : rw.n), dim3(128), 0, s,
                   static_cast<const T *>(b.zx), b.ld, inner, static_cast<T *>(b.xbc), static_cast<T *>(b.conv_state), rw, conv_w, conv_b, ch, d.conv);
    SMC_LAUNCH_CHECK(ctx);
    if (seq && rw.n > 1) {
        smc_launch_dep(ctx->use_pdl, ssm_conv_keep_kernel<T>, dim3((ch + 127) / 128, d.conv < rw.n ? d.conv : rw.n), dim3(128), 0, s,
                       static_cast<const T *>(b.zx), b.ld, inner, static_cast<T *>(b.conv_state), rw, ch, d.conv);
        SMC_LAUNCH_CHECK(ctx);
    }
    const size_t smem = ((size_t)2 * SC * d.state + SC * 16 + 2 * SC) * sizeof(float);
    const dim3 grid(d.heads, (d.vdim + 15) / 16, seq ? 1 : rw.n);
#define SMC_SCAN(NP)                                                                                                                              \
    do {                                                                                                                                          \
        if (smem > 40 * 1024)                                                                                                                     \
            SMC_CUDA(ctx, cudaFuncSetAttribute(ssm_scan_kernel<T, NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));                  \
        smc_launch_dep(ctx->use_pdl, ssm_scan_kernel<T, NP>, grid, dim3(128), smem, s, (const T *)b.xbc, b.dt_raw, b.y, b.state, rw, dt_bias,      \
                       a_log, d_skip, d.heads, d.vdim, d.state, d.groups);                                                                        \
    } while (0)
    if (d.state <= 32) SMC_SCAN(4);
    else if (d.state <= 64) SMC_SCAN(8);
    else if (d.state <= 128) SMC_SCAN(16);
    else if (d.state <= 256) SMC_SCAN(32);
    else SMC_SCAN(64);
#undef SMC_SCAN
    SMC_LAUNCH_CHECK(ctx);
    const size_t nsm = (size_t)(inner / d.norm_groups) * sizeof(float);
    if (nsm > 40 * 1024) SMC_CUDA(ctx, cudaFuncSetAttribute(ssm_gate_norm_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)nsm));
    smc_launch_dep(ctx->use_pdl, ssm_gate_norm_kernel<T>, dim3(rw.n, d.norm_groups), dim3(128), nsm, s, (const float *)b.y, static_cast<const T *>(b.zx),
                   b.ld, norm, static_cast<T *>(b.o), inner, d.norm_groups, d.eps);
    SMC_LAUNCH_CHECK(ctx);
    return SMC_OK;
}

}  // namespace

size_t smc_ssm_work_floats(const smc_ssm_dims &, int) { return 0; }

int smc_ssm_mix(smc_ctx *ctx, const smc_ssm_dims &d, const smc_ssm_bufs &b, const smc_rows &rw, int is_bf16, const float *conv_w, const float *conv_b,
                const float *dt_bias, const float *a_log, const float *d_skip, const float *norm, int pos0, cudaStream_t s)
{
    (void)pos0;
    if (is_bf16) return mix<bf16>(ctx, d, b, rw, conv_w, conv_b, dt_bias, a_log, d_skip, norm, s);
    return mix<float>(ctx, d, b, rw, conv_w, conv_b, dt_bias, a_log, d_skip, norm, s);
}
